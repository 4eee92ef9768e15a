"""Small layer-stack configurations and helpers shared by their tests."""
import numpy as np

from oracle import bavutar_oracle as bo
from oracle import layer_stack_oracle as lo


def oracle(config):
    """The plain implementation of a configuration's family."""
    return {"Keselix": lo, "Bavutar": bo}[config["architecture"]]


def attn(heads=3, dim=20, rot=6, vdim=12, rank=28, window=9, base=500.0, scale=0.3, ff=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale,
                      "mask": {"size": window}, "rot": {"base": base, "dims": rot}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def ssm(inner=52, state=5, conv=4, rank=3, ff=None):
    return {"type": "mamba1", "mixer": {"inner": inner, "state": state, "conv": conv, "dt_rank": rank},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def model(layers, width=72, vocab=131, loop=None, mult=0.45, eps=1e-3):
    return {"architecture": "Keselix", "vocab": vocab, "width": width, "layers": layers, "loop": loop,
            "norm": {"eps": eps}, "residual_mult": mult}


CONFIGS = {
    # sizes that are no multiples of 8, a state-space layer with and an attention layer without a feed-forward
    "odd": model([ssm(ff=44), attn(), ssm(inner=30, state=9, conv=2, rank=11)], loop={"start": 0, "stop": 2, "times": 2}),
    # several 64-column blocks per head, a window over many tiles, a loop that runs once
    "wide": model([attn(heads=4, dim=96, rot=32, vdim=128, rank=64, window=150, ff=256), ssm(inner=256, state=16, rank=8)],
                  width=128, vocab=300, loop={"start": 1, "stop": 2, "times": 1}, eps=1e-5),
    # one head, the largest blocks of the tensor-core attention, no convolution history, no loop
    "tall": model([attn(heads=1, dim=130, rot=8, vdim=200, rank=160, window=70), ssm(inner=64, state=40, conv=1, rank=16),
                   attn(heads=9, dim=8, rot=2, vdim=72, rank=8, window=1, ff=24)], width=64, vocab=77),
    # key rows beyond the tensor-core attention's sizes
    "fat": model([ssm(inner=96, state=70, conv=3, rank=5), attn(heads=2, dim=260, rot=64, vdim=40, rank=600, window=33, scale=0.06, ff=80)],
                 width=96, vocab=140, loop={"start": 1, "stop": 2, "times": 3}),
}


# ------------------------------------------------------------------ Bavutar ----
def gqa(heads=6, kv_heads=2, dim=20, vdim=12, scale=0.25, temp=(0.5, 7), kv_from=None, ff=44):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def delta(heads=3, kv_heads=1, dim=20, vdim=12, conv=3, ff=36):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def ssd(heads=6, vdim=5, state=9, groups=3, norm_groups=2, conv=4, ff=None):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups,
                                        "conv": conv}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def bavutar(layers, width=72, vocab=131, alpha=1.4, eps=1e-3, scale=1.5, cap=9.0):
    return {"architecture": "Bavutar", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}, "postln_alpha": alpha,
            "embedding": {"scale": scale}, "logit_softcap": cap}


BAVUTAR = {
    # sizes that are no multiples of 8, key heads shared by several heads, a layer without a feed-forward, keys and
    # values taken from a layer two steps back under another scale and without a temperature
    "odd": bavutar([delta(), gqa(), ssd(), gqa(kv_from=1, scale=0.4, temp=None, ff=None), delta(heads=4, kv_heads=2, dim=9, vdim=7)]),
    # sizes of whole tiles, no cap, one head group, as many norm parts as heads
    "wide": bavutar([gqa(heads=8, kv_heads=2, dim=128, vdim=96, scale=0.09, temp=(0.2, 64), ff=256),
                     delta(heads=4, kv_heads=4, dim=128, vdim=64, conv=4, ff=128),
                     ssd(heads=8, vdim=32, state=64, groups=1, norm_groups=8, ff=128),
                     gqa(heads=8, kv_heads=2, dim=128, vdim=96, scale=0.09, temp=(0.6, 50), kv_from=0, ff=256)],
                    width=128, vocab=300, eps=1e-5, cap=None),
    # one query head, the largest blocks of the tensor-core attention, no convolution history, large states
    "tall": bavutar([gqa(heads=1, kv_heads=1, dim=200, vdim=250, scale=0.07, temp=(1.0, 1)),
                     delta(heads=2, kv_heads=2, dim=150, vdim=40, conv=1),
                     ssd(heads=2, vdim=70, state=200, groups=2, norm_groups=1, conv=6)], width=64, vocab=77, alpha=1.0, scale=1.0),
    # heads beyond the tensor-core attention's sizes, more query heads per key head than one block takes, long taps
    "fat": bavutar([gqa(heads=4, kv_heads=4, dim=300, vdim=20, scale=0.06), gqa(heads=20, kv_heads=1, dim=16, vdim=16),
                    delta(heads=1, kv_heads=1, dim=256, vdim=300, conv=5), ssd(heads=3, vdim=64, state=128, groups=1, norm_groups=3, conv=2)],
                   width=96, vocab=140, alpha=2.0),
}


# (dtype, prompt rows from which the tensor-core path is taken)
PATHS = {"f32": ("float32", 0), "few_rows": ("bfloat16", 1 << 20), "many_rows": ("bfloat16", 2)}
# root mean square over the vocabulary of the logit difference, relative to the logits' own spread
TOL = {"f32": 2e-5, "few_rows": 2e-2, "many_rows": 4e-2}


def weights(config, seed=0, **kw):
    return oracle(config).random_weights(config, seed, **kw)


def tensors(w):
    import torch
    return {k: torch.from_numpy(np.ascontiguousarray(v)).to(torch.bfloat16) for k, v in w.items()}


def network(config, w, path="f32", seq=512, **over):
    """A CausalTransformer of the configuration over the CUDA library."""
    from mesh_transformer import registry
    from mesh_transformer.transformer_shard import CausalTransformer
    dtype, tc_rows = PATHS[path]
    cfg = registry.prepare(dict(config, mtj_dtype=dtype, mtj_tc_min_rows=tc_rows, seq=seq, **over))
    cfg = registry.family(cfg).fit_tensors(cfg, {k: v.shape for k, v in w.items()})
    net = CausalTransformer(cfg, init_weights=False)
    net.state = {"params": registry.family(cfg).state_from_tensors(cfg, tensors(w)), "step": np.array(0)}
    return net


def runtime(config, w, path="f32", seq=512, max_batch=1, max_gen=1, max_rows=None):
    from mesh_transformer._runtime import ShardRuntime
    net = network(config, w, path, seq)
    rt = ShardRuntime(net.config, max_batch=max_batch, max_gen=max_gen, max_rows=max_rows)
    rt.load_params(net.state["params"])
    return rt


def ids(seed, n, vocab):
    return np.random.default_rng(seed).integers(0, vocab, n).astype(np.int32)


def extend(rt, slot, toks, want=None):
    import torch
    t = torch.tensor(np.asarray(toks, np.int32), device=rt.device)
    return rt.extend(slot, t, range(len(toks)) if want is None else want).cpu().numpy()


def error(got, want):
    """Worst relative rms error over positions (means taken off: a common shift of the logits means nothing)."""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(-1, keepdims=True)
    return float(np.sqrt((d * d).mean(-1)).max() / (want - want.mean(-1, keepdims=True)).std())


def position_errors(got, want):
    """The relative rms error of every position."""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / (want - want.mean(-1, keepdims=True)).std()


def agrees(errors, path):
    """Errors of many positions within the path's tolerance: all of them in 32-bit; with bf16 operands 95 in a hundred,
    and none beyond three times it (the norm of a recurrence's nearly empty output, or a score at a near-tie, magnifies the
    rounding of its operands at single positions)."""
    e = np.asarray(errors).reshape(-1)
    return e.max() <= TOL[path] if path == "f32" else np.quantile(e, 0.95) <= TOL[path] and e.max() <= 3 * TOL[path]


def greedy_agrees(got, config, w, prompt, margin):
    """Greedy ids equal the oracle's; a difference is accepted only at a near-tie of the oracle's own logits (and ends
    the comparison, the sequences differ from there on)."""
    toks = list(prompt)
    for t in got:
        last = oracle(config).forward(config, w, toks)[-1]
        best = int(len(last) - 1 - np.argmax(last[::-1]))
        if int(t) != best:
            assert last[best] - last[int(t)] <= margin * last.std(), (int(t), best, last[best] - last[int(t)])
            return
        toks.append(best)
