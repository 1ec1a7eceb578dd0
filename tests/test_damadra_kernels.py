"""Damadra's mechanisms alone, with inputs made so that a fault shows: one key that holds almost all of a query's weight, at page
borders and one token inside and outside the window; tables of distance biases in which one bucket stands out, with borders that
are whole numbers and tables longer than shared memory takes; keys whose sizes before the norm differ by factors, so that values
taken after the norm would show; experts that are never chosen, identities only.  References: `plain_damadra.py`.

The mixers are built alone, with identity matrices as their input projections, so that a row given to the mixer IS its row of
queries, keys and values, and what `forward_unprojected` returns is compared before the output projection."""

import numpy as np
import pytest
import torch

import plain_damadra as pd
from test_fakelorn_kernels import MixerAlone, _dev, _i32, _rounded

pytestmark = pytest.mark.gpu
F64 = torch.float64
DTYPES = [torch.float32, torch.bfloat16]
EPS = 1e-5
NAMES = {"q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm"}


class AttentionAlone(MixerAlone):
    def load(self, part, tensors):
        infos = {}
        for p in (part,) + tuple(part.children()):
            infos.update(p.param_infos())
        assert set(infos) == {"m." + k for k in tensors}
        placed = {"m." + k: _dev(t, torch.float32 if infos["m." + k].kind == "scalars" else self.rt.dtype) for k, t in tensors.items()}
        for p in (part,) + tuple(part.children()):
            p.load(placed)


class Case:
    """A mixer of one of the two kinds: its library parameters, its tensors and its plain counterpart."""

    def __init__(self, windowed, shape, rel, far, scale, window=0, temp=(0.0, 1), seed=0, own=True):
        H, G, dim, vd = shape
        assert not windowed or vd == dim
        self.windowed, self.window, self.own = windowed, window, own
        self.m = {"heads": H, "kv_heads": G, "dim": dim, "vdim": vd, "scale": scale, "bias_max": far, "q_temp": {"coef": temp[0], "every": temp[1]}, "mask": {"size": window}}
        rng = np.random.default_rng(seed)
        a, b = H * dim, (H + G) * dim
        self.cols = b + (0 if windowed else G * vd)
        eye = np.eye(self.cols)
        bf = lambda x: _rounded(x, torch.bfloat16).numpy()  # noqa: E731
        t = {"q": eye[:a], "o": np.zeros((self.cols, H * vd)), "rel": bf(rel), "q.norm": bf(1 + 0.1 * rng.standard_normal(a if windowed else dim))}
        if own:
            t.update({"k": eye[a:b], "k.norm": bf(1 + 0.1 * rng.standard_normal(b - a if windowed else dim))})
            if not windowed:
                t["v"] = eye[b:]
        self.tensors, self.W = t, {k: torch.as_tensor(v) for k, v in t.items()}
        from rusty_llama_b200.spec import PartSpec

        self.params = {"hidden_size": self.cols, "num_heads": H, "num_kv_heads": G, "head_dim": dim, "value_dim": vd, "scale": scale, "window": window, "qk_norm": EPS,
                       "position": PartSpec("distance_bias", {"num_heads": H, "max_distance": far}, "m."), "names": NAMES, "own_kv": own}
        if windowed:
            self.params.update(values="keys", qk_norm_span="all")
        else:
            self.params["q_temperature"] = temp

    def alone(self, dtype, **kw):
        return AttentionAlone("attention", self.params, self.tensors, dtype, **kw)

    def keys_values(self, rows):
        return pd.windowed_queries_keys_values(rows, self.W, "", self.m, EPS)[1:] if self.windowed else pd.full_keys_values(rows, self.W, "", self.m, EPS)

    def plain(self, rows, kv=None, window=None):
        """What goes into the output projection; kv: another layer's keys and values; window: another window."""
        rows = torch.as_tensor(rows)
        k, v = self.keys_values(rows) if kv is None else kv
        q = pd.windowed_queries_keys_values(rows, self.W, "", self.m, EPS)[0] if self.windowed else pd.full_queries(rows, self.W, "", self.m, EPS)
        bias = pd.bias_matrix(self.W["rel"], self.m["bias_max"], len(rows))
        return pd.softmax_attention(q, k, v, self.m["scale"], bias, self.window if window is None else window).reshape(len(rows), -1)


def check_cuts(mixer, rows, ref, dtype, cut_lists, tol_bf, what=""):
    L, top = len(rows), float(ref.abs().max())
    tol = 2e-5 if dtype == torch.float32 else tol_bf
    whole = mixer.run(rows, [L])
    worst = (whole - ref).abs().max(1).values
    assert float(worst.max()) <= tol * top, f"{what}: {float(worst.max()) / top:.2e} of the range, row {int(worst.argmax())}"
    for cuts in cut_lists:
        got = mixer.run(rows, cuts)
        worst = (got - ref).abs().max(1).values
        assert float(worst.max()) <= tol * top, f"{what}, cuts {cuts}: {float(worst.max()) / top:.2e} of the range, row {int(worst.argmax())}"
        if dtype == torch.float32:
            assert torch.equal(got, whole), f"{what}, cuts {cuts}: other bits"


# heads, kv heads, key size (and value size): sizes of the general kernel, of the padded tensor-core kernels, of the tcgen05 and TMA ones
WINDOWED = [(6, 2, 12), (3, 1, 7), (4, 2, 56), (2, 2, 72), (4, 2, 64), (12, 1, 64), (3, 1, 128), (4, 4, 136)]
FULL = [(3, 1, 10, 12), (4, 2, 56, 40), (5, 5, 96, 64), (6, 3, 40, 24), (4, 2, 64, 64), (9, 1, 64, 64), (2, 1, 128, 128), (2, 2, 24, 200), (3, 1, 32, 128), (8, 2, 128, 40)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", WINDOWED)
def test_one_key_inside_and_outside_the_window_and_values_before_the_norm(shape, dtype):
    """The key of token `target` fits every query and no other key does: the last query that the window lets see it and the first that it
    does not differ by nearly all of their weight.  Every token's key has another length, which the norm takes away from the scores
    and which the values keep.  As one prompt, in portions, and one by one."""
    H, G, dim = shape
    L = 270
    for case, (window, target) in enumerate([(64, 63), (65, 64), (1, 40), (100, 27), (130, 127), (33, 200)]):
        rng = np.random.default_rng(10 * H + case)
        c = Case(True, (H, G, dim, dim), 0.5 * rng.standard_normal((12, H)), 90, 9.0 / dim, window, seed=case)
        u = rng.standard_normal(dim)
        u /= np.linalg.norm(u)
        q = 1.2 * u + 0.05 * rng.standard_normal((L, H, dim))
        k = rng.standard_normal((L, G, dim))
        k -= (k @ u)[..., None] * u
        k[target] = 1.5 * u
        k *= rng.uniform(0.4, 2.5, (L, 1, 1))
        rows = _rounded(np.concatenate([q.reshape(L, -1), k.reshape(L, -1)], axis=1), dtype).numpy()
        ref = c.plain(rows)
        if window > 1:
            e, i = target + window, target + window - 1
            assert float((c.plain(rows, window=window + 1) - ref)[e].abs().max()) > 0.2 * float(ref[e].abs().max())
            assert float((c.plain(rows, window=window - 1) - ref)[i].abs().max()) > 0.2 * float(ref[i].abs().max())
        check_cuts(c.alone(dtype), rows, ref, dtype, ([2, 61, 2, 100, 33], [target + 1], []), 3e-2, f"window {window}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", FULL)
def test_one_key_far_away_and_a_reader_of_the_same_keys(shape, dtype):
    """One key among hundreds, at page borders and at the start, under a temperature that grows; a second layer with queries, biases and
    constants of its own reads the same keys and values without writing any."""
    from rusty_llama_b200.parts import MIXERS
    from rusty_llama_b200.spec import PartSpec

    H, G, dim, vd = shape
    L = 330
    for target in (63, 64, 0):
        rng = np.random.default_rng(target + H)
        c = Case(False, shape, 0.5 * rng.standard_normal((20, H)), 200, 8.0 / dim, temp=(0.1, 20), seed=target)
        r = Case(False, shape, 0.8 * rng.standard_normal((6, H)), 40, 6.0 / dim, temp=(0.4, 64), seed=target + 1, own=False)
        u = rng.standard_normal(dim)
        u /= np.linalg.norm(u)
        q = 1.2 * u + 0.05 * rng.standard_normal((L, H, dim))
        k = rng.standard_normal((L, G, dim))
        k -= (k @ u)[..., None] * u
        k[target] = 1.5 * u
        rows = _rounded(np.concatenate([x.reshape(L, -1) for x in (q, k, rng.standard_normal((L, G, vd)))], axis=1), dtype).numpy()
        mixer = c.alone(dtype)
        reader = MIXERS.build(PartSpec("attention", r.params, "m."), mixer.rt)
        mixer.load(reader, r.tensors)
        assert reader.cache_need() is None
        kv = c.keys_values(torch.as_tensor(rows))
        refs = [c.plain(rows), r.plain(rows, kv=kv)]
        s = mixer.cache.open_sequence()
        got, at = [[], []], 0
        for n in [100, 2, 62, 130] + [1] * (L - 294):
            for g, o in zip(got, mixer.step([s], [rows[at : at + n]], readers=[reader])):
                g.append(o[0])
            at += n
        mixer.cache.close_sequence(s)
        for who, g, ref in zip(("own", "reader"), got, refs):
            worst = (torch.cat(g) - ref).abs().max(1).values
            tol = 2e-5 if dtype == torch.float32 else 3e-2
            assert float(worst.max()) <= tol * float(ref.abs().max()), f"{who}, target {target}: row {int(worst.argmax())}"
        check_cuts(mixer, rows, refs[0], dtype, ([], [300]), 3e-2, f"target {target}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", FULL)
def test_one_bucket_of_distances_stands_out(shape, dtype):
    """Scores near zero and one bucket's bias of 9: a query's result is the mean of the values at that bucket's distances, so a border that
    is one token off shows.  Tables whose borders are whole numbers, of two rows, and one too long for shared memory."""
    H, G, dim, vd = shape
    L = 300
    for case, (rows_n, far, bucket) in enumerate([(16, 128, 7), (16, 128, 8), (16, 128, 10), (16, 128, 15), (2, 100, 1), (40, 60000, 22), (8, 300, 0)]):
        rng = np.random.default_rng(case)
        rel = np.zeros((rows_n, H))
        rel[bucket] = 9.0
        rel[:, H - 1] *= -1.0  # the last head: everything but that bucket
        c = Case(False, shape, rel, far, 1e-3 / dim, seed=case)
        rows = _rounded(rng.standard_normal((L, c.cols)), dtype).numpy()
        ref = c.plain(rows)
        check_cuts(c.alone(dtype), rows, ref, dtype, ([2, 61, 2, 100, 33], []) if case % 2 else ([],), 2e-2, f"bucket {bucket} of {rows_n} up to {far}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", [(4, 2, 64, 64), (6, 2, 128, 128), (10, 5, 40, 24), (24, 2, 64, 64)])
@pytest.mark.parametrize("windowed", [True, False])
def test_batches_of_unequal_sequences(windowed, shape, dtype):
    """Four sequences of unequal lengths as one batch of prompts and then one token each (the decode kernels with several sequences and
    the key range in parts), each against itself alone; pages of closed sequences are used again."""
    H, G, dim, vd = shape
    vd = dim if windowed else vd
    rng = np.random.default_rng(dim)
    c = Case(windowed, (H, G, dim, vd), rng.standard_normal((14, H)), 120, 2.5 / np.sqrt(dim), 150 if windowed else 0, temp=(0.5, 30), seed=3)
    mixer = c.alone(dtype, max_tokens=64 * 14)
    lens, extra = (1, 64, 200, 321), 5
    seqs = [_rounded(rng.standard_normal((n + extra, c.cols)), dtype).numpy() for n in lens]
    for again in range(2):
        slots = [mixer.cache.open_sequence() for _ in lens]
        got = [[o] for o in mixer.step(slots, [s[:n] for s, n in zip(seqs, lens)])]
        for j in range(extra):
            for g, o in zip(got, mixer.step(slots, [s[n + j : n + j + 1] for s, n in zip(seqs, lens)])):
                g.append(o)
        for s in slots:
            mixer.cache.close_sequence(s)
        for rows, g, n in zip(seqs, got, lens):
            ref, g = c.plain(rows), torch.cat(g)
            tol = 2e-5 if dtype == torch.float32 else 4e-2
            assert float((g - ref).abs().max()) <= tol * float(ref.abs().max()), f"pass {again}, length {n}"
            if dtype == torch.float32:
                assert torch.equal(g, mixer.run(rows, [n]))
        seqs = seqs[::-1]
        lens = lens[::-1]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", [(4, 2, 56, 40), (6, 2, 128, 128), (4, 1, 64, 96), (3, 3, 136, 40), (4, 2, 12, 10)])
def test_a_bias_beside_caps_sinks_windows_and_chunks(shape, dtype):
    """The bias is added after the cap; the other options of the attention keep their meaning beside it.  Prompts and single tokens."""
    from rusty_llama_b200.parts.attention import chunked_attention_runner
    from types import SimpleNamespace

    H, G, kd, vd = shape
    rng = np.random.default_rng(kd)
    n, L = 200, 17
    q, k, v = (_rounded(rng.standard_normal(s), dtype) for s in ((n, H, kd), (n, G, kd), (n, G, vd)))
    table = _rounded(rng.standard_normal((H, L)), torch.float32)
    sink = _rounded(rng.standard_normal(H), torch.float32)
    pages = [3, 0, 2, 1]
    kp, vp = (torch.zeros((4, G, 64, size), dtype=dtype, device="cuda") for size in (kd, vd))
    for i in range(n):
        kp[pages[i // 64], :, i % 64], vp[pages[i // 64], :, i % 64] = _dev(k[i], dtype), _dev(v[i], dtype)
    gap = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    for window, chunk, cap, use_sink in ((0, 0, 2.0, True), (70, 0, 0.0, True), (0, 48, 1.5, False), (33, 96, 0.0, False)):
        scale = 1.5 / np.sqrt(kd)
        s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(H // G, 1)) * scale
        s = (cap * torch.tanh(s / cap) if cap else s) + table[:, gap.clamp(0, L - 1)]
        vis = (gap >= 0) & ((gap < window) if window else True)
        if chunk:
            vis = vis & (torch.arange(n)[:, None] // chunk == torch.arange(n)[None, :] // chunk)
        e = torch.exp(s.masked_fill(~vis[None], -np.inf))
        den = e.sum(-1, keepdim=True) + (torch.exp(sink)[:, None, None] if use_sink else 0.0)
        ref = torch.einsum("hij,jhv->ihv", e / den, v.repeat_interleave(H // G, 1)).reshape(n, -1)
        for p0, m in ((0, n), (130, 70), (199, 1), (64, 1)):
            step = SimpleNamespace(tok_seq=_i32(np.zeros(m)), tok_pos=_i32(np.arange(p0, p0 + m)), seq_start=_i32([0, m]), seq_pos0=_i32([p0]), max_q_len=m, n_seqs=1,
                                   decode_only=m == 1)
            rows = torch.zeros((m, H * kd + 8), dtype=dtype, device="cuda")
            rows[:, : H * kd] = _dev(q[p0 : p0 + m].reshape(m, -1), dtype)
            got = chunked_attention_runner(rows, kp, vp, _i32([pages]), step, H, G, kd, vd, scale, chunk, cap, _dev(sink, torch.float32) if use_sink else None,
                                           window=window, bias=_dev(table, torch.float32))().to(F64).cpu()
            tol = 1e-5 if dtype == torch.float32 else 2.5e-2
            worst = (got - ref[p0 : p0 + m]).abs().max(1).values
            assert float(worst.max()) <= tol * float(ref.abs().max()), f"window {window}, chunk {chunk}, cap {cap}, from {p0}: row {int(worst.argmax())}"


# ------------------------------------------------------------------ norms, temperature, storing
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,kd,vd", [(4, 2, 56, 40), (3, 1, 10, 6), (2, 2, 128, 128), (5, 1, 40, 8), (8, 4, 64, 64), (1, 1, 256, 16), (40, 8, 128, 128)])
def test_rows_normed_tempered_and_stored(H, G, kd, vd, dtype):
    """Norms over all heads at once and head by head, in rows whose heads differ by factors; values that are the raw keys; the
    temperature around its steps; rows of queries only leave the pages alone."""
    from rusty_llama_b200.kernels import ops

    T = 9
    rng = np.random.default_rng(H + kd)
    pos = np.array([0, 5, 6, 7, 62, 63, 64, 127, 190])
    table = [[2, 0, 1]]
    for whole, keys in ((True, True), (True, False), (False, False)):
        if keys:
            vd = kd
        cols = (H + G) * kd + (0 if keys else G * vd)
        x = rng.standard_normal((T, cols))
        x[:, : (H + G) * kd] *= np.repeat(rng.uniform(0.2, 4.0, (T, H + G)), kd, axis=1)
        x = _rounded(x, dtype)
        wq, wk = (_rounded(1 + 0.3 * rng.standard_normal((n if whole else 1) * kd), torch.bfloat16) for n in (H, G))
        norm = (lambda t, w: pd.rms(t.reshape(T, -1), EPS) * w) if whole else (lambda t, w: (pd.rms(t, EPS) * w).reshape(T, -1))
        temp = pd.query_temperature(torch.as_tensor(pos), 0.7, 7)
        q, k = x[:, : H * kd].reshape(T, H, kd), x[:, H * kd : (H + G) * kd].reshape(T, G, kd)
        want_q, want_k = norm(q, wq) * temp[:, None], norm(k, wk)
        want_v = k.reshape(T, -1) if keys else x[:, (H + G) * kd :]
        args = (_i32(pos), _i32(np.zeros(T)), _i32(table))
        kw = dict(q_norm=_dev(wq, torch.float32), norm_eps=EPS, norm_whole=whole, temperature=(0.7, 7))
        rows = _dev(x, dtype)
        kp, vp = (torch.zeros((3, G, 64, n), dtype=dtype, device="cuda") for n in (kd, vd))
        ops.qkv_prep(rows, None, *args, kp, vp, None, 1.0, H, G, kd, vd, 0, False, k_norm=_dev(wk, torch.float32), v_from_k=keys, **kw)
        got_k, got_v = (torch.stack([p[table[0][n // 64], :, n % 64].reshape(-1) for n in pos]).to(F64).cpu() for p in (kp, vp))
        tol = 2e-6 if dtype == torch.float32 else 4.5e-3  # one rounding
        for name, got, want in (("q", rows[:, : H * kd].to(F64).cpu(), want_q), ("k", got_k, want_k), ("v", got_v, want_v)):
            assert float(((got - want).abs() / (want.abs() + 1e-3)).max()) <= tol, f"{name}, whole={whole}"
        only_q = _dev(x[:, : H * kd].contiguous(), dtype)
        ops.qkv_prep(only_q, None, *args[:2], None, None, None, None, 1.0, H, 0, kd, vd, 0, False, **kw)
        assert torch.equal(only_q, rows[:, : H * kd])


# ------------------------------------------------------------------ experts and identities
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E,identity,top,d,ff,T", [(5, 2, 3, 64, 40, 9), (4, 3, 2, 128, 72, 200), (1, 2, 3, 68, 30, 7), (3, 0, 1, 96, 24, 150), (12, 5, 3, 192, 80, 333), (2, 6, 4, 36, 17, 40)])
def test_experts_beside_choices_that_hand_the_input_on(E, identity, top, d, ff, T, dtype):
    from rusty_llama_b200.parts import FEED_FORWARDS, Runtime
    from rusty_llama_b200.spec import PartSpec

    rng = np.random.default_rng(E * 100 + d)
    params = {"hidden_size": d, "n_experts": E, "identity": identity, "top": top, "expert_ff": ff, "bias": True, "renormalize": False, "activation": "relu2"}
    for lean in (0.0, 5.0, -5.0):  # the corrections leave the choice open, force the identities, or keep them out
        corr = 0.05 * rng.standard_normal(E + identity)
        corr[E:] += lean
        W = {"router": rng.standard_normal((E + identity, d)) / np.sqrt(d), "correction": corr}
        for e in range(E):
            W[f"e{e}.up"], W[f"e{e}.down"] = rng.standard_normal((ff, d)) / np.sqrt(d), rng.standard_normal((d, ff)) / np.sqrt(ff)
        W = {k: _rounded(v, torch.bfloat16) for k, v in W.items()}
        part = FEED_FORWARDS.build(PartSpec("routed_experts", params, "f."), Runtime.create("cuda:0", dtype))
        infos = part.param_infos()
        assert set(infos) == {"f." + k for k in W}
        part.load({"f." + k: _dev(v, torch.float32 if infos["f." + k].kind == "scalars" else dtype) for k, v in W.items()})
        x = _rounded(1.3 * rng.standard_normal((T, d)), dtype)
        want = pd.moe_ff(x, W, "", {"experts": E, "identity": identity, "top": top})
        chosen = pd.route(x, W, "", top)[0]
        if identity >= top and lean > 0:
            assert bool((chosen >= E).all())
        if E >= top and lean < 0:
            assert bool((chosen < E).all())
        got = part.forward(_dev(x, dtype), None).to(F64).cpu()
        tol = 1e-5 if dtype == torch.float32 else 1.5e-2
        worst = (got - want).abs().max(1).values
        assert float(worst.max()) <= tol * float(want.abs().max()), f"lean {lean}: row {int(worst.argmax())}"


def test_pairs_without_an_expert_have_no_rows():
    from rusty_llama_b200.kernels import ops

    ids = [[0, 5], [3, 4], [1, 0], [5, 4], [1, 3]]
    order, place, tiles, _ = ops.moe_plan(_i32(ids), 4, 32)
    place, tiles = place.tolist(), tiles.tolist()
    assert [p < 0 for p in place] == [i >= 4 for row in ids for i in row]
    assert tiles[0] == 3 and [tiles[1 + 3 * i : 4 + 3 * i] for i in range(3)] == [[0, 0, 2], [1, 2, 2], [3, 4, 2]]
    flat = [i for row in ids for i in row]
    assert all(order.tolist()[p] == i for i, p in enumerate(place) if p >= 0) and sorted(p for p in place if p >= 0) == list(range(sum(i < 4 for i in flat)))


# ------------------------------------------------------------------ results normed behind their sublayer, the stream read as it is
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,d", [(3, 96), (70, 256), (5, 70), (130, 4096), (2, 6000), (67, 1028)])
def test_the_stream_is_read_as_it_is_and_results_are_normed_and_scaled(T, d, dtype):
    from rusty_llama_b200.parts import NORMS, ResidualStream, Runtime
    from rusty_llama_b200.spec import PartSpec

    rt = Runtime.create("cuda:0", dtype)
    read = NORMS.build(PartSpec("identity"), rt)
    behind = NORMS.build(PartSpec("rmsnorm", {"size": d, "eps": EPS, "factor": 0.3}, "n."), rt)
    rng = np.random.default_rng(d)
    w = _rounded(1 + 0.3 * rng.standard_normal(d), torch.bfloat16)
    assert behind.param_infos()["n.weight"].kind == "scalars"
    behind.load({"n.weight": _dev(w, torch.float32)})
    x0, parts = rng.standard_normal((T, d)), rng.standard_normal((3, T, d))
    stream = ResidualStream(_dev(x0, torch.float32), dtype)
    tol = 1e-6 if dtype == torch.float32 else 4e-3
    x = _rounded(x0, torch.float32)
    first = read.forward(stream)
    assert first.dtype == dtype and torch.equal(first.to(F64).cpu(), x.to(dtype).to(F64)) and torch.equal(stream.x.to(F64).cpu(), x)
    # a normed result, as partial sums in 32-bit and as one row in the activation type; then a plain result
    for delta in (_dev(parts, torch.float32), _dev(parts[0], dtype)):
        stream.add(delta, norm=behind.rms_weight())
        y = read.forward(stream)
        s = delta.to(F64).cpu()
        x = x + pd.rms(s.sum(0) if s.dim() == 3 else s, EPS) * w * 0.3
        assert float((stream.x.to(F64).cpu() - x).abs().max()) <= 2e-6 * float(x.abs().max())
        assert torch.equal(y, stream.x.to(dtype))
    stream.add(_dev(parts[1], dtype))
    rows = _i32([T - 1, 0])
    y = read.forward(stream, rows=rows)
    x = x + _rounded(parts[1], dtype)
    assert tuple(y.shape) == (2, d) and float((y.to(F64).cpu() - x[[T - 1, 0]]).abs().max()) <= tol * float(x.abs().max())
