"""Bavutar models on the GPU against the plain oracle: each mechanism alone, prompts, portions, token by token, batches,
slots used again, far keys at page borders, chunk edges of the recurrences, first tokens, long decoding, generation,
serving and trace replay."""
import json
import os
import subprocess
import threading

import numpy as np
import pytest

from oracle import bavutar_oracle as bo
from tests import stack_util as su
from tests.test_bavutar_cpu import marker_model

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module")
def cases(cuda_device):
    """{config: (config, weights, ids, oracle logits, oracle residuals)} of one 200-token sequence each."""
    out = {}
    for i, (name, cfg) in enumerate(sorted(su.BAVUTAR.items())):
        w = su.weights(cfg, 20 + i)
        toks = su.ids(40 + i, 200, cfg["vocab"])
        out[name] = (cfg, w, toks) + bo.forward(cfg, w, toks, return_layers=True)
    return out


@pytest.mark.parametrize("path", sorted(su.PATHS))
@pytest.mark.parametrize("name", sorted(su.BAVUTAR))
def test_prompts_portions_and_tokens(cases, name, path):
    """The same sequence as one prompt, in portions of many sizes, and token by token: every position's logits against
    the oracle, and the residual stream after every layer."""
    import torch
    cfg, w, toks, want, trail = cases[name]
    rt = su.runtime(cfg, w, path, seq=220, max_rows=220)
    dev = torch.tensor(toks, device=rt.device)
    for run in range(len(trail)):
        got = rt.stack_residual(dev, run + 1).cpu().numpy()
        d = np.abs(got - trail[run]).max() / trail[run].std()
        assert d <= {"f32": 1e-4, "few_rows": 0.15, "many_rows": 0.3}[path], (run, d)
    rt.start_batch(1)
    errs = {"whole": su.position_errors(su.extend(rt, 0, toks), want)}
    for sizes in ((2,), (3, 2, 17, 64, 1, 5), (1,), (129, 2, 31), (63, 1, 65, 16)):
        rt.release(0)
        at, i, got = 0, 0, []
        while at < len(toks):
            n = min(sizes[i % len(sizes)], len(toks) - at)
            got.append(su.extend(rt, 0, toks[at:at + n]))
            at, i = at + n, i + 1
        errs[sizes] = su.position_errors(np.concatenate(got), want)
    rt.check_device_status()
    rt.close()
    for sizes, e in errs.items():
        assert su.agrees(e, path), (sizes, e.max())


@pytest.mark.parametrize("layers", [[su.gqa(ff=None)], [su.gqa(temp=None, ff=None), su.gqa(kv_from=0, scale=0.5, ff=None)], [su.delta(ff=None)],
                                    [su.ssd()], [su.ssd(ff=50)], [su.gqa(ff=30)],
                                    [su.delta(heads=1, kv_heads=1, dim=1, vdim=1, conv=1)], [su.ssd(heads=1, vdim=1, state=1, groups=1, norm_groups=1, conv=1)],
                                    [su.gqa(heads=1, kv_heads=1, dim=1, vdim=1)]])
def test_each_mechanism_alone(cuda_device, layers):
    """Few layers, with an eps that matters, in 32-bit: the residual stream itself."""
    import torch
    cfg = su.bavutar(layers, eps=0.2)
    w = su.weights(cfg, 1, ranks=(3, 9))
    toks = su.ids(1, 50, cfg["vocab"])
    logits, trail = bo.forward(cfg, w, toks, return_layers=True)
    rt = su.runtime(cfg, w, "f32")
    for run in range(len(layers)):
        got = rt.stack_residual(torch.tensor(toks, device=rt.device), run + 1).cpu().numpy()
        assert np.abs(got - trail[run]).max() <= 2e-5 * np.abs(trail[run]).max()
    rt.start_batch(1)
    assert su.error(su.extend(rt, 0, toks), logits) <= su.TOL["f32"]
    rt.close()


@pytest.mark.parametrize("path", sorted(su.PATHS))
def test_far_keys_and_page_borders(cuda_device, path):
    """A key that outweighs all others, anywhere from the first token to the query's neighbour, at page, tile and portion
    borders, for query tiles' edges and decoded tokens."""
    for heads, kv_heads, dim in ((4, 2, 16), (3, 3, 80), (18, 1, 16)):
        cfg, w = marker_model(heads, kv_heads, dim)
        rt = su.runtime(cfg, w, path, seq=400, max_rows=300)
        rt.start_batch(1)
        for q in (1, 63, 64, 65, 127, 128, 255, 257, 330):
            toks = 3 + np.arange(q + 3) % 30
            toks[q] = 1
            for key in {0, 1, 15, 16, 62, 63, 64, 127, 128, q - 1} - set(range(q, 400)):
                marked = toks.copy()
                marked[key] = 2
                want = bo.forward(cfg, w, marked)[q:q + 1]
                for cut in (len(marked), q, max(q - 1, 1), max(key, 1), key + 1):
                    rt.release(0)
                    su.extend(rt, 0, marked[:min(cut, q)], want=())
                    got = su.extend(rt, 0, marked[min(cut, q):])
                    e = su.error(got[q - min(cut, q)][None], want)
                    assert e <= su.TOL[path], (heads, dim, q, key, cut, e)
        rt.check_device_status()
        rt.close()


@pytest.mark.parametrize("path", sorted(su.PATHS))
def test_state_across_every_cut(cuda_device, path):
    """Slow decays, so that a state lost or applied twice at any cut shows: a long prompt cut once at every place around
    the tiles of the scans, and continued token by token."""
    for layer in (su.delta(heads=4, kv_heads=2, dim=64, vdim=32, conv=4), su.ssd(heads=4, vdim=32, state=64, groups=2, conv=4)):
        cfg = su.bavutar([layer], eps=1e-5)
        w = su.weights(cfg, 9)
        w["l0.mix.A_log"] = np.full_like(w["l0.mix.A_log"], -3.0)
        toks = su.ids(9, 160, cfg["vocab"])
        want = bo.forward(cfg, w, toks)
        rt = su.runtime(cfg, w, path, seq=200)
        rt.start_batch(1)
        for cut in (1, 2, 3, 4, 15, 16, 17, 31, 32, 33, 63, 64, 65, 127, 128, 129, 158):
            rt.release(0)
            got = np.concatenate([su.extend(rt, 0, toks[:cut]), su.extend(rt, 0, toks[cut:cut + 1]), su.extend(rt, 0, toks[cut + 1:])])
            assert su.error(got, want) <= su.TOL[path], (layer["type"], cut)
        rt.check_device_status()
        rt.close()


@pytest.mark.parametrize("path", sorted(su.PATHS))
def test_extreme_decays(cuda_device, path):
    """Heads that forget at once beside heads that never forget, in one chunk."""
    for layer in (su.delta(heads=4, kv_heads=4, dim=32, vdim=32), su.ssd(heads=4, vdim=32, state=32, groups=4)):
        cfg = su.bavutar([layer], eps=1e-5)
        w = su.weights(cfg, 10)
        w["l0.mix.A_log"] = np.array([-12.0, -4.0, 2.0, 5.0], np.float32)
        toks = su.ids(10, 300, cfg["vocab"])
        rt = su.runtime(cfg, w, path, seq=320)
        rt.start_batch(1)
        assert su.error(su.extend(rt, 0, toks), bo.forward(cfg, w, toks)) <= su.TOL[path], layer["type"]
        rt.check_device_status()
        rt.close()


def test_many_heads_and_sequences(cuda_device):
    """More column groups than the GPU has SMs, so that blocks of the chunked scans hold four of them: unequal prompts
    prefilled together, then a few decoded tokens, against each alone."""
    import torch
    for layer in (su.delta(heads=20, kv_heads=5, dim=40, vdim=64, ff=None), su.ssd(heads=20, vdim=60, state=48, groups=4, norm_groups=5)):
        cfg = su.bavutar([layer], eps=1e-3)
        w = su.weights(cfg, 13)
        lens, seq, steps = [90, 33, 70, 2], 90, 3
        seqs = [su.ids(80 + i, n + steps, cfg["vocab"]) for i, n in enumerate(lens)]
        want = [bo.forward(cfg, w, s)[n - 1:] for s, n in zip(seqs, lens)]
        rt = su.runtime(cfg, w, "many_rows", seq=seq, max_batch=4, max_gen=steps + 1, max_rows=4 * seq)
        ctx = np.zeros((4, seq), np.int32)
        for b, n in enumerate(lens):
            ctx[b, seq - n:] = seqs[b][:n]
        rt.prefill(torch.tensor(ctx, device=rt.device), lens)
        logits, errs = torch.empty((4, cfg["vocab"]), device=rt.device), []
        for t in range(steps + 1):
            feed = None if t == 0 else torch.tensor([s[n - 1 + t] for s, n in zip(seqs, lens)], dtype=torch.int32, device=rt.device)
            rt.decode_step(feed, None, logits)
            errs += [su.error(logits.cpu().numpy()[b:b + 1], want[b][t:t + 1]) for b in range(4)]
        rt.check_device_status()
        rt.close()
        assert max(errs) <= 2 * su.TOL["many_rows"], (layer["type"], errs)


@pytest.mark.parametrize("path", sorted(su.PATHS))
def test_query_temperature_at_its_steps(cuda_device, path):
    """Queries right before and after the positions where the temperature changes, in prompts and decoded."""
    cfg = su.bavutar([su.gqa(temp=(2.0, 33), scale=0.4)], eps=1e-5)
    w = su.weights(cfg, 12)
    toks = su.ids(12, 140, cfg["vocab"])
    want = bo.forward(cfg, w, toks)
    rt = su.runtime(cfg, w, path, seq=160)
    rt.start_batch(1)
    assert su.error(su.extend(rt, 0, toks), want) <= su.TOL[path]
    for step in (32, 65, 98):
        rt.release(0)
        su.extend(rt, 0, toks[:step - 1], want=())
        got = np.concatenate([su.extend(rt, 0, [t]) for t in toks[step - 1:step + 3]])
        assert su.error(got, want[step - 1:step + 3]) <= su.TOL[path]
    rt.close()


@pytest.mark.parametrize("path", sorted(su.PATHS))
def test_one_call_longer_than_a_chunk(cases, path):
    """The library cuts a long call itself, at max_rows; wanted places in any order across the cuts."""
    cfg, w, toks, want, _ = cases["odd"]
    rt = su.runtime(cfg, w, path, max_rows=33)
    rt.start_batch(1)
    order = [199, 0, 32, 33, 66, 65, 100, 1, 198]
    assert su.error(su.extend(rt, 0, toks, order), want[order]) <= su.TOL[path]
    rt.close()


@pytest.mark.parametrize("path", sorted(su.PATHS))
def test_first_tokens(cases, path):
    """Sequences of 1, 2, 3 ... tokens, each fresh in a slot that has held another."""
    cfg, w, toks, want, _ = cases["odd"]
    rt = su.runtime(cfg, w, path)
    rt.start_batch(1)
    for n in range(1, 8):
        su.extend(rt, 0, su.ids(n, 30, cfg["vocab"]), want=())
        rt.release(0)
        assert su.error(su.extend(rt, 0, toks[:n]), want[:n]) <= su.TOL[path]
        rt.release(0)
        got = np.concatenate([su.extend(rt, 0, [t]) for t in toks[:n]])
        assert su.error(got, want[:n]) <= su.TOL[path]
        rt.release(0)
    rt.close()


@pytest.mark.parametrize("path,batch", [("f32", 3), ("few_rows", 1), ("many_rows", 5)])
def test_long_decoding(cuda_device, path, batch):
    """Hundreds of decode steps through the replayed step graph; every sequence of the batch against the oracle, at
    positions all along the way."""
    import torch
    cfg = su.bavutar([su.delta(), su.gqa(temp=(0.3, 50)), su.ssd(), su.gqa(kv_from=1)], eps=3e-2)
    w = su.weights(cfg, 8)
    n = 420
    toks = np.stack([su.ids(60 + b, n, cfg["vocab"]) for b in range(batch)])
    want = [bo.forward(cfg, w, toks[b]) for b in range(batch)]
    rt = su.runtime(cfg, w, path, seq=16, max_batch=batch, max_gen=n, max_rows=16)
    rt.start_batch(batch)
    logits = torch.empty((batch, cfg["vocab"]), device=rt.device)
    got = np.empty((batch, n, cfg["vocab"]))
    for t in range(n):
        rt.decode_step(torch.tensor(toks[:, t], device=rt.device), None, logits)
        got[:, t] = logits.cpu().numpy()
    rt.check_device_status()
    rt.close()
    for b in range(batch):
        assert su.agrees(su.position_errors(got[b], want[b]), path), b


@pytest.mark.parametrize("name", ["odd", "wide"])
@pytest.mark.parametrize("path", sorted(su.PATHS))
def test_batches_of_unequal_requests(cases, path, name):
    """Left-padded prompts of very different lengths prefilled together, then decoded together, against each alone;
    the padding ids do not matter."""
    import torch
    cfg, w, _, _, _ = cases[name]
    seq, lens, steps = 96, [96, 1, 2, 50, 17], 12
    seqs = [su.ids(70 + i, n + steps, cfg["vocab"]) for i, n in enumerate(lens)]
    want = [bo.forward(cfg, w, s)[n - 1:] for s, n in zip(seqs, lens)]
    for rows in (seq, 40, 5 * seq):
        rt = su.runtime(cfg, w, path, seq=seq, max_batch=5, max_gen=steps + 1, max_rows=rows)
        ctx = np.zeros((5, seq), np.int32)
        for b, n in enumerate(lens):
            ctx[b, :seq - n] = 77
            ctx[b, seq - n:] = seqs[b][:n]
        rt.prefill(torch.tensor(ctx, device=rt.device), lens)
        logits, errs = torch.empty((5, cfg["vocab"]), device=rt.device), []
        for t in range(steps + 1):
            feed = None if t == 0 else torch.tensor([s[n - 1 + t] for s, n in zip(seqs, lens)], dtype=torch.int32, device=rt.device)
            rt.decode_step(feed, None, logits)
            got = logits.cpu().numpy()
            for b in range(5):
                errs.append(su.error(got[b:b + 1], want[b][t:t + 1]))
        assert su.agrees(errs, "many_rows" if path == "few_rows" else path), (rows, max(errs))   # five rows decode on the tensor cores
        rt.check_device_status()
        rt.close()


def test_interleaved_requests_in_slots(cases):
    """Requests that come and go in three slots, their portions interleaved: bit for bit what each gives alone."""
    cfg, w, toks, want, _ = cases["wide"]
    rt = su.runtime(cfg, w, "many_rows", seq=256, max_batch=3)
    rt.start_batch(3)
    reqs = {i: (toks[i:i + 60 + 30 * i], (7, 1, 33, 2)) for i in range(5)}

    def portions(i):
        t, sizes = reqs[i]
        at, k = 0, 0
        while at < len(t):
            n = min(sizes[(k + i) % 4], len(t) - at)
            yield t[at:at + n]
            at, k = at + n, k + 1

    alone = {}
    for i in reqs:
        alone[i] = np.concatenate([su.extend(rt, i % 3, p) for p in portions(i)])
        rt.release(i % 3)
    live, waiting, got, free = {}, [3, 1, 4, 0, 2], {i: [] for i in reqs}, [2, 0, 1]
    while waiting or live:
        while waiting and free:
            i = waiting.pop(0)
            live[i] = (free.pop(0), portions(i))
        for i in list(live):
            slot, it = live[i]
            p = next(it, None)
            if p is None:
                rt.release(slot)
                free.append(slot)
                del live[i]
            else:
                got[i].append(su.extend(rt, slot, p))
    for i in reqs:
        assert np.array_equal(np.concatenate(got[i]), alone[i]), i
    rt.close()


@pytest.mark.parametrize("path", sorted(su.PATHS))
def test_greedy_generation_through_the_network(cases, path):
    """CausalTransformer.generate: unequal left-padded prompts, greedy, against the oracle's greedy continuation."""
    cfg, w, toks, _, _ = cases["odd"]
    net = su.network(cfg, w, path, seq=48)
    for lens in ([48], [5, 48, 1, 20]):
        ctx = np.zeros((len(lens), 48), np.uint32)
        for b, n in enumerate(lens):
            ctx[b, 48 - n:] = toks[b:b + n]
        _, out = net.generate(ctx, lens, 10, {"top_p": np.zeros(len(lens)), "temp": np.ones(len(lens))}, return_logits=True)
        for b, n in enumerate(lens):
            su.greedy_agrees(out[0][b, :, 0], cfg, w, toks[b:b + n], 2 * su.TOL[path])
            full = bo.forward(cfg, w, list(toks[b:b + n]) + [int(t) for t in out[0][b, :-1, 0]])
            assert su.error(out[2][b, :, 0], full[n - 1:]) <= su.TOL[path]
    net.close()


def test_sampled_generation_equals_the_sampler_on_the_same_logits(cases):
    from mesh_transformer.sampling import nucleaus_sample
    from oracle import sampling_oracle
    cfg, w, toks, _, _ = cases["odd"]
    net = su.network(dict(cfg, sampler=nucleaus_sample), w, "few_rows", seq=32)
    ctx = np.stack([toks[:32], toks[32:64]]).astype(np.uint32)
    un = np.random.default_rng(5).random((6, 2, cfg["vocab"]), dtype=np.float32).clip(sampling_oracle.TINY, None)
    _, out = net.generate(ctx, [32, 9], 6, {"top_p": np.array([0.9, 0.7]), "temp": np.array([0.8, 1.3])}, return_logits=True,
                          uniforms=un)
    for t in range(6):
        for b, (p, temp) in enumerate(((0.9, 0.8), (0.7, 1.3))):
            ids = sampling_oracle.nucleaus_sample(un[t][b:b + 1], out[2][b:b + 1, t, 0], np.float32(p), np.float32(temp))
            assert int(ids[0]) == int(out[0][b, t, 0])
    net.close()


def test_eval_loss(cases):
    cfg, w, toks, want, _ = cases["odd"]
    net = su.network(cfg, w, "many_rows", seq=200)
    lse = np.log(np.exp(want - want.max(-1, keepdims=True)).sum(-1)) + want.max(-1)
    loss = lse[:-1] - want[np.arange(199), toks[1:]]
    r = net.eval({"obs": np.stack([toks[:-1]] * 2), "target": np.stack([toks[1:]] * 2)})
    assert np.abs(r["all_loss"] - loss[None]).max() <= 0.25 and abs(r["loss"].mean() - loss.mean()) <= 2e-2
    net.close()


def test_continuous_batching_service(cases):
    """Requests join a running batch: prompts admitted between decode steps into slots that earlier requests have
    left, greedy completions against the oracle's."""
    import serve
    from mesh_transformer.sampling import nucleaus_sample
    cfg, w, _, _, _ = cases["odd"]
    net = su.network(dict(cfg, sampler=nucleaus_sample), w, "f32", seq=32)

    class Tok:
        def encode(self, text):
            return [b % cfg["vocab"] for b in text.encode()]

        def decode(self, out):
            return [int(i) for i in out]

    svc = serve.ContinuousBatchingService(net, Tok(), seq=32, slots=3, gen_length=7, epoch_steps=25)
    loop = threading.Thread(target=svc.serve_forever)
    loop.start()
    texts = ["a", "some words", "one more request that is longer than the context", "xy", "state", "0123456789", "zz top"]
    answers = [None] * len(texts)

    def client(i):
        answers[i] = svc.complete({"context": texts[i], "top_p": 0.0, "temp": 1.0})

    clients = [threading.Thread(target=client, args=(i,)) for i in range(len(texts))]
    for c in clients:
        c.start()
    for c in clients:
        c.join(timeout=60)
    svc.stop()
    loop.join(timeout=60)
    for text, a in zip(texts, answers):
        assert a is not None
        su.greedy_agrees(a["completion"], cfg, w, Tok().encode(text)[-32:], 1e-4)
    net.close()


def test_trace_replay(cases, tmp_path):
    """bin/trace_run on a model folder: portions, wanted places, finished requests."""
    from mesh_transformer.checkpoint import write_safetensors
    cfg, w, toks, want, _ = cases["odd"]
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(tmp_path / "model.safetensors", su.tensors(w))
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:30].tolist(), "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[30:33].tolist(), "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[33:34].tolist(), "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": toks[:5].tolist(), "want": [4, 1]}], "end": ["b"]}]
    out = tmp_path / "out"
    out.mkdir()
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    p = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "64"], input="\n".join(map(json.dumps, steps)) + "\n", capture_output=True, text=True,
                       timeout=300)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.split("\n") if l.startswith("done")] == [f"done {i}" for i in range(4)]
    read = lambda i: np.fromfile(out / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"])
    assert not (out / "1.f32").exists()
    for i, at in ((0, [0, 29]), (2, [33]), (3, [4, 1])):
        assert su.error(read(i), want[at]) <= su.TOL["f32"]
