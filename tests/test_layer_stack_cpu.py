"""Layer-stack models without a GPU: configuration, tensor names, model folders, and checks of the oracle itself --
each mechanism against an independent form, and that the inputs the GPU tests use show a planted mistake."""
import json

import numpy as np
import pytest

from oracle import layer_stack_oracle as lo
from tests import stack_util as su


@pytest.fixture(scope="module", autouse=True)
def built():
    import __graft_entry__ as ge
    ge.build()


@pytest.mark.parametrize("name", sorted(su.CONFIGS))
def test_tensor_names_and_shapes(name):
    from mesh_transformer import layer_stack, registry
    cfg = registry.prepare(su.CONFIGS[name])
    registry.family(cfg).validate(cfg)
    assert layer_stack.tensor_shapes(cfg) == lo.tensor_shapes(su.CONFIGS[name])
    assert registry.prepare(cfg) == cfg


def test_registry_picks_families_and_rejects_what_it_cannot_run():
    from mesh_transformer import registry
    assert registry.names() == ["Bavutar", "Keselix", "gptj"]
    assert registry.family({}).__name__ == "GptJ"
    with pytest.raises(NotImplementedError):
        registry.family({"architecture": "no such design"})
    bad = [dict(su.CONFIGS["odd"], cores_per_replica=2), dict(su.CONFIGS["odd"], mtj_dtype="float16"),
           dict(su.CONFIGS["odd"], layers=[dict(su.ssm(), type="other")]),
           dict(su.CONFIGS["odd"], layers=[dict(su.ssm(), mlp={"kind": "sparse", "ff": 8})]),
           dict(su.CONFIGS["odd"], loop={"start": 1, "stop": 9, "times": 2})]
    for cfg in bad:
        with pytest.raises((NotImplementedError, ValueError)):
            registry.family(cfg).validate(registry.prepare(cfg))


def test_library_rejects_bad_stacks_with_a_message():
    import ctypes
    from mesh_transformer import _lib, registry
    caps = dict(rank=0, max_batch=1, max_gen=4, max_rows=32)
    h = ctypes.c_void_p()
    for layer in (su.attn(window=0), su.attn(rot=3), su.attn(rank=5000), su.ssm(state=1000), su.ssm(conv=0)):
        cfg = registry.prepare(su.model([layer]))
        assert registry.family(cfg).create(cfg, caps, ctypes.byref(h)) != 0
        assert b"layer 0" in _lib.lib.mtj_last_error()
    cfg = registry.prepare(su.CONFIGS["odd"])
    assert registry.family(cfg).create(cfg, caps, ctypes.byref(h)) == 0
    assert _lib.lib.mtj_weights_bytes(h) > 0 and _lib.lib.mtj_workspace_bytes(h) > 0
    assert _lib.lib.mtj_decode_step(h, None, None, None, None, 1, None, None, None) != 0     # nothing bound yet
    assert _lib.lib.mtj_destroy(h) == 0


def test_model_folder_round_trip(tmp_path):
    import torch
    from mesh_transformer import registry
    from mesh_transformer.checkpoint import read_safetensors, write_safetensors
    cfg = su.CONFIGS["odd"]
    t = su.tensors(su.weights(cfg, 5))
    write_safetensors(tmp_path / "model.safetensors", dict(t, table=torch.arange(6, dtype=torch.int32).reshape(2, 3)))
    back = read_safetensors(tmp_path / "model.safetensors")
    assert back.pop("table").tolist() == [[0, 1, 2], [3, 4, 5]]
    assert all(torch.equal(back[k], t[k]) for k in t)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    read = registry.read_config(str(tmp_path), seq=99)
    assert read["n_vocab"] == cfg["vocab"] and read["seq"] == 99
    fam = registry.family(read)
    assert set(fam.state_from_tensors(read, back)["layer_stack"]) == set(t)
    with pytest.raises(ValueError, match="missing"):
        fam.state_from_tensors(read, {k: v for k, v in back.items() if k != "embed"})
    with pytest.raises(ValueError, match="shape"):
        fam.state_from_tensors(read, dict(back, embed=back["embed"][:-1]))


# ------------------------------------------------------------------- the oracle ----
def test_rotation_depends_on_distance_only_and_pairs_neighbours():
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal((1, 6)), rng.standard_normal((1, 6))
    dot = lambda p, r: float((lo.rotate_interleaved(q, [p], 50.0) @ lo.rotate_interleaved(k, [r], 50.0).T)[0, 0])
    assert abs(dot(7, 3) - dot(104, 100)) < 1e-9 and abs(dot(7, 3) - dot(8, 3)) > 1e-3
    x = np.zeros((1, 6))
    x[0, 2] = 1.0
    r = lo.rotate_interleaved(x, [1], 50.0)[0]
    a = 50.0 ** (-2.0 / 6)
    assert np.allclose(r, [0, 0, np.cos(a), np.sin(a), 0, 0])


def test_attention_equals_its_absorbed_form():
    """Scores against the latent with W_uk folded into the query, values from the attended latent."""
    m = su.attn()["mixer"]
    rng = np.random.default_rng(1)
    T, d, H, n, r, v, R = 30, 40, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    w = {"q": rng.standard_normal((H * (n + r), d)), "dkv": rng.standard_normal((R + r, d)), "dkv.norm": rng.standard_normal(R),
         "uk": rng.standard_normal((H * n, R)), "uv": rng.standard_normal((H * v, R)), "o": rng.standard_normal((d, H * v))}
    h = rng.standard_normal((T, d)) * 0.3
    pos = np.arange(T)
    q = (h @ w["q"].T).reshape(T, H, n + r)
    down = h @ w["dkv"].T
    c = lo.rms_norm(down[:, :R], w["dkv.norm"], 1e-3)
    kr = lo.rotate_interleaved(down[:, R:], pos, m["rot"]["base"])
    qr = lo.rotate_interleaved(q[..., n:], pos, m["rot"]["base"])
    qa = np.einsum("thn,hnr->thr", q[..., :n], w["uk"].reshape(H, n, R))
    s = (np.einsum("thr,jr->htj", qa, c) + np.einsum("thr,jr->htj", qr, kr)) * m["scale"]
    dist = pos[:, None] - pos[None, :]
    s = np.where((dist >= 0) & (dist < m["mask"]["size"]), s, -np.inf)
    p = np.exp(s - s.max(-1, keepdims=True))
    p /= p.sum(-1, keepdims=True)
    o = np.einsum("hvr,thr->thv", w["uv"].reshape(H, v, R), np.einsum("htj,jr->thr", p, c)).reshape(T, H * v)
    assert np.allclose(o @ w["o"].T, lo.latent_attention(h, w, m, 1e-3))


def test_scan_equals_its_unrolled_sum_and_conv_its_definition():
    rng = np.random.default_rng(2)
    T, C, N = 12, 4, 3
    u, dt, A = rng.standard_normal((T, C)), rng.uniform(0.01, 1, (T, C)), -rng.uniform(0.1, 3, (C, N))
    B, Cm, D = rng.standard_normal((T, N)), rng.standard_normal((T, N)), rng.standard_normal(C)
    y = lo.selective_scan(u, dt, A, B, Cm, D)
    t = T - 1
    want = D * u[t]
    for s in range(T):
        decay = np.exp(dt[s + 1:].sum(0)[:, None] * A)
        want = want + (decay * (dt[s] * u[s])[:, None] * B[s][None]) @ Cm[t]
    assert np.allclose(y[t], want)
    x, k, b = rng.standard_normal((5, 2)), rng.standard_normal((2, 3)), rng.standard_normal(2)
    got = lo.causal_conv(x, k, b)
    assert np.allclose(got[0], x[0] * k[:, 2] + b)
    assert np.allclose(got[4], x[2] * k[:, 0] + x[3] * k[:, 1] + x[4] * k[:, 2] + b)


def test_layer_schedule():
    layers = [None] * 4
    assert lo.layer_schedule({"layers": layers}) == [(i, False) for i in range(4)]
    got = lo.layer_schedule({"layers": layers, "loop": {"start": 1, "stop": 3, "times": 2}})
    assert got == [(0, False), (1, True), (2, False), (1, True), (2, False), (3, False)]


def _changed(cfg, change):
    cfg = json.loads(json.dumps(cfg))
    change(cfg)
    return cfg


@pytest.mark.parametrize("fault", ["window", "eps", "mult", "base", "scale", "times"])
def test_random_models_show_a_wrong_constant(fault):
    """The random weights of the GPU tests are such that a wrong constant moves the logits by more than the bf16
    tolerance."""
    cfg = _changed(su.CONFIGS["odd"], lambda c: c["norm"].update(eps=0.05))
    w = su.weights(cfg, 3)
    toks = su.ids(3, 60, cfg["vocab"])
    mix = lambda c: c["layers"][1]["mixer"]
    other = _changed(cfg, {
        "window": lambda c: mix(c)["mask"].update(size=mix(c)["mask"]["size"] + 1),
        "eps": lambda c: c["norm"].update(eps=0.1),
        "mult": lambda c: c.update(residual_mult=c["residual_mult"] * 1.3),
        "base": lambda c: mix(c)["rot"].update(base=mix(c)["rot"]["base"] * 3),
        "scale": lambda c: mix(c).update(scale=mix(c)["scale"] * 1.3),
        "times": lambda c: c["loop"].update(times=1)}[fault])
    assert su.error(lo.forward(other, w, toks), lo.forward(cfg, w, toks)) > 4e-2


def test_lost_state_shows_long_after():
    """A recurrent state dropped in the middle of a sequence is visible 40 tokens later."""
    cfg = su.model([su.ssm()])
    w = su.weights(cfg, 4)
    toks = su.ids(4, 80, cfg["vocab"])
    whole = lo.forward(cfg, w, toks)
    cut = lo.forward(cfg, w, toks[40:])
    assert su.error(cut[-1:], whole[-1:]) > 4e-2


def marker_model(window, rank=24, heads=2, rot=4, dim=16, gain=12.0):
    """One attention layer in which token 1, as a query, scores token 2's key far above every other: its output
    shows at once whether a key at a given distance is visible.  Tokens 3 .. are the background."""
    cfg = su.model([su.attn(heads=heads, dim=dim, rot=rot, vdim=20, rank=rank, window=window, scale=1.0)], width=64, vocab=40,
                   mult=1.0, eps=1e-5)
    w = su.weights(cfg, 11)
    rng = np.random.default_rng(12)
    e = np.linalg.qr(rng.standard_normal((64, 40)))[0].T * 8.0          # orthogonal rows of unit rms
    w["embed"] = lo.to_bf16_grid(e)
    w["l0.norm1"] = np.ones_like(w["l0.norm1"])
    q = np.zeros_like(w["l0.mix.q"])
    q[::dim + rot] = e[1] / 64 * gain                                    # first dimension of every head
    w["l0.mix.q"] = lo.to_bf16_grid(q)
    dkv = 0.2 * np.asarray(w["l0.mix.dkv"])
    dkv[0] = e[2] / 64 * 20.0
    dkv[rank:] = 0.0
    w["l0.mix.dkv"] = lo.to_bf16_grid(dkv)
    w["l0.mix.dkv.norm"] = np.ones_like(w["l0.mix.dkv.norm"])
    uk = np.zeros_like(w["l0.mix.uk"])
    uk[::dim, 0] = 1.0
    w["l0.mix.uk"] = uk
    return cfg, w


def test_marker_model_shows_one_key():
    cfg, w = marker_model(window=9)
    toks = np.full(40, 5)
    toks[3:] = 3 + np.arange(37) % 30
    base = toks.copy()
    base[20] = 1
    inside, outside = base.copy(), base.copy()
    inside[20 - 8], outside[20 - 9] = 2, 2
    ref, a, b = (lo.forward(cfg, w, t)[20] for t in (base, inside, outside))
    scale = ref.std()
    assert np.sqrt(np.mean((a - ref) ** 2)) > 0.3 * scale and np.sqrt(np.mean((b - ref) ** 2)) < 1e-9 * scale
