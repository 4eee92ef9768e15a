"""Small layer-stack configurations and helpers shared by their tests."""
import numpy as np

from oracle import layer_stack_oracle as lo


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

# (dtype, prompt rows from which the tensor-core path is taken)
PATHS = {"f32": ("float32", 0), "few_rows": ("bfloat16", 1 << 20), "many_rows": ("bfloat16", 2)}
# root mean square over the vocabulary of the logit difference, relative to the logits' own spread
TOL = {"f32": 2e-5, "few_rows": 2e-2, "many_rows": 4e-2}


def weights(config, seed=0, **kw):
    return lo.random_weights(config, seed, **kw)


def tensors(w):
    import torch
    return {k: torch.from_numpy(np.ascontiguousarray(v)).to(torch.bfloat16) for k, v in w.items()}


def network(config, w, path="f32", seq=512, **over):
    """A CausalTransformer of the configuration over the CUDA library."""
    from mesh_transformer import registry
    from mesh_transformer.transformer_shard import CausalTransformer
    dtype, tc_rows = PATHS[path]
    cfg = registry.prepare(dict(config, mtj_dtype=dtype, mtj_tc_min_rows=tc_rows, seq=seq, **over))
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


def greedy_agrees(got, config, w, prompt, margin):
    """Greedy ids equal the oracle's; a difference is accepted only at a near-tie of the oracle's own logits (and ends
    the comparison, the sequences differ from there on)."""
    toks = list(prompt)
    for t in got:
        last = lo.forward(config, w, toks)[-1]
        best = int(len(last) - 1 - np.argmax(last[::-1]))
        if int(t) != best:
            assert last[best] - last[int(t)] <= margin * last.std(), (int(t), best, last[best] - last[int(t)])
            return
        toks.append(best)
