"""Fakelorn's mechanisms alone, with inputs made so that a fault shows: one key in one map of a head that holds almost all of that
map's weight, at page borders and one token inside and outside the window; one latent among hundreds; a state that is written
once and read hundreds of tokens later at every chunk border; decays that forget at once and decays that never do; norms whose
parts differ by factors of ten.  References: `plain_fakelorn.py`.

The mixers are built alone, with identity matrices as their input projections, so that a row given to the mixer IS its row of
queries, keys and values, and what `forward_unprojected` returns is compared before the output projection."""

import numpy as np
import pytest
import torch

import plain_fakelorn as pf
from test_parts import ctx_for

pytestmark = pytest.mark.gpu
F64 = torch.float64
DTYPES = [torch.float32, torch.bfloat16]


def _dev(a, dtype):
    return torch.as_tensor(np.asarray(a, dtype=np.float64)).to("cuda", dtype)


def _rounded(a, dtype):
    return torch.as_tensor(np.asarray(a, dtype=np.float64)).to(dtype).to(F64)


def _i32(a):
    return torch.tensor(np.asarray(a), dtype=torch.int32, device="cuda")


class MixerAlone:
    """A mixer part with a cache of its own; sequences are fed rows in portions."""

    def __init__(self, kind, params, tensors, dtype, max_tokens=64 * 40, max_seqs=4, need=None):
        from rusty_llama_b200.cache import Cache
        from rusty_llama_b200.parts import MIXERS, Runtime
        from rusty_llama_b200.spec import PartSpec

        self.rt = Runtime.create("cuda:0", dtype)
        self.part = MIXERS.build(PartSpec(kind, params, "m."), self.rt)
        self.load(self.part, tensors)
        self.cache = Cache([(0, need or self.part.cache_need())], max_tokens, max_seqs, dtype, "cuda:0")
        self.dtype = dtype

    def load(self, part, tensors):
        infos = part.param_infos()
        assert set(infos) == {"m." + k for k in tensors}
        placed = {}
        for k, t in tensors.items():
            info = infos["m." + k]
            assert tuple(info.shape) == tuple(t.shape), k
            placed["m." + k] = _dev(t, torch.float32 if info.kind == "scalars" else self.rt.dtype)
        part.load(placed)

    def step(self, slots, rows, readers=()):
        """rows: one [n, d] array per slot; returns one [n, out] float64 tensor per slot (with readers: a list per part)."""
        lens = [len(r) for r in rows]
        pos0 = [self.cache.length(s) for s in slots]
        ctx, tables = ctx_for(self.cache, slots, pos0, lens)
        x = _dev(np.concatenate([np.asarray(r) for r in rows]), self.dtype)
        outs = []
        for part, shared in [(self.part, False)] + [(r, True) for r in readers]:
            a, _ = part.forward_unprojected(x, ctx, self.cache.view(0, tables), shared)
            outs.append([t.to(F64).cpu() for t in torch.split(a, lens)])
        self.cache.commit(slots, lens)
        self.cache.check_consistent()
        return outs if readers else outs[0]

    def run(self, rows, cuts):
        s = self.cache.open_sequence()
        out, at = [], 0
        for n in list(cuts) + [1] * (len(rows) - sum(cuts)):
            out.append(self.step([s], [rows[at : at + n]])[0])
            at += n
        self.cache.close_sequence(s)
        return torch.cat(out)


# ------------------------------------------------------------------ differential attention
def _differential(shape, dtype, window, scale, diff, eps, seed, **kw):
    H, G, dim, vd = shape
    cols = H * 2 * dim + G * (2 * dim + vd)
    rng = np.random.default_rng(seed)
    eye = np.eye(cols)
    lam = {n: _rounded(rng.standard_normal(dim) / np.sqrt(dim), torch.bfloat16).numpy() for n in ("lq1", "lk1", "lq2", "lk2")}
    a, b = H * 2 * dim, H * 2 * dim + G * 2 * dim
    tensors = dict(q=eye[:a], k=eye[a:b], v=eye[b:], o=np.zeros((cols, H * vd)), **lam)
    params = {"hidden_size": cols, "num_heads": H, "num_kv_heads": G, "map_dim": dim, "value_dim": vd, "scale": scale, "window": window, "diff": diff, "eps": eps,
              "names": {"q": "q", "k": "k", "v": "v", "o": "o"}}
    return MixerAlone("differential_attention", params, tensors, dtype, **kw), {k: torch.as_tensor(v) for k, v in lam.items()}


def _plain_differential(q, k, v, lam, scale, window, diff, eps):
    T, H = q.shape[0], q.shape[1]
    a1, a2 = pf.differential_maps(q, k, v, scale, window)
    return pf.combine_maps(a1, a2, pf.lambda_of(lam, "", diff), diff, eps).reshape(T, -1)


SHAPES = [(6, 2, 10, 12), (4, 2, 32, 64), (3, 1, 64, 128), (10, 5, 24, 40), (8, 1, 32, 64), (2, 2, 16, 72), (1, 1, 12, 24)]
WINDOWS = [(64, 63), (65, 64), (1, 40), (100, 27), (0, 0), (130, 127)]  # (window, the token whose key stands out)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", SHAPES)
def test_one_key_of_one_map_inside_and_outside_the_window(shape, dtype):
    """The key of token `target` fits every query in map 1 or in map 2, every other score is near zero: the last query that the window
    lets see it and the first that it does not differ by nearly all of that map's weight.  As one prompt, in portions, and one by one."""
    H, G, dim, vd = shape
    L, scale, diff, eps = 270, 1.0, 0.3, 1e-5
    for case, (window, target) in enumerate(WINDOWS):
        mixer, lam = _differential(shape, dtype, window, scale, diff, eps, seed=case)
        rng = np.random.default_rng(100 * H + case)
        m = case % 2
        q, k, v = (_rounded(x, dtype) for x in (0.02 * rng.standard_normal((L, H, 2, dim)), 0.02 * rng.standard_normal((L, G, 2, dim)), rng.standard_normal((L, G, vd))))
        unit = rng.standard_normal(dim)
        unit = _rounded(4.5 * unit / np.linalg.norm(unit), dtype)
        q[:, :, m] = _rounded((q[:, :, m] + unit).numpy(), dtype)
        k[target, :, m] = unit
        rows = torch.cat([q.reshape(L, -1), k.reshape(L, -1), v.reshape(L, -1)], dim=1).numpy()
        ref = _plain_differential(q, k, v, lam, scale, window, diff, eps)
        top = float(ref.abs().max())
        if window > 1 and target + window < L:  # a window that is one token off would show
            wider = _plain_differential(q, k, v, lam, scale, window + 1, diff, eps)
            narrower = _plain_differential(q, k, v, lam, scale, window - 1, diff, eps)
            assert float((wider - ref)[target + window].abs().max()) > 0.2 * top and float((narrower - ref)[target + window - 1].abs().max()) > 0.2 * top
        tol = 2e-5 if dtype == torch.float32 else 4e-2
        whole = mixer.run(rows, [L])
        assert float((whole - ref).abs().max()) <= tol * top, f"window {window}: {float((whole - ref).abs().max()) / top:.2e}, first row {int((whole - ref).abs().max(1).values.argmax())}"
        for cuts in ([2, 61, 2, 100, 33], [target + 1], []):
            got = mixer.run(rows, cuts)
            assert float((got - ref).abs().max()) <= tol * top, f"window {window}, cuts {cuts}: row {int((got - ref).abs().max(1).values.argmax())}"
            if dtype == torch.float32:
                assert torch.equal(got, whole), f"window {window}, cuts {cuts}: other bits"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", [(4, 2, 32, 64), (6, 2, 64, 128), (10, 5, 24, 40)])
def test_differential_batches_of_unequal_sequences(shape, dtype):
    """Four sequences of unequal lengths as one batch of prompts and then one token each (the decode kernels with several sequences and
    the key range in parts), each against itself alone."""
    H, G, dim, vd = shape
    window, scale, diff, eps = 150, 0.4, 0.6, 1e-6
    mixer, lam = _differential(shape, dtype, window, scale, diff, eps, seed=1)
    rng = np.random.default_rng(dim)
    lens, extra = (1, 64, 200, 321), 5
    seqs = []
    for n in lens:
        q, k, v = (_rounded(rng.standard_normal(s), dtype) for s in ((n + extra, H, 2, dim), (n + extra, G, 2, dim), (n + extra, G, vd)))
        seqs.append((q, k, v, torch.cat([x.reshape(n + extra, -1) for x in (q, k, v)], dim=1).numpy()))
    slots = [mixer.cache.open_sequence() for _ in lens]
    got = [[o] for o in mixer.step(slots, [s[3][:n] for s, n in zip(seqs, lens)])]
    for j in range(extra):
        for g, o in zip(got, mixer.step(slots, [s[3][n + j : n + j + 1] for s, n in zip(seqs, lens)])):
            g.append(o)
    for s in slots:
        mixer.cache.close_sequence(s)
    for (q, k, v, rows), g, n in zip(seqs, got, lens):
        ref = _plain_differential(q, k, v, lam, scale, window, diff, eps)
        g = torch.cat(g)
        tol = 2e-5 if dtype == torch.float32 else 5e-2
        assert float((g - ref).abs().max()) <= tol * float(ref.abs().max())
        if dtype == torch.float32:
            assert torch.equal(g, mixer.run(rows, [n]))


# ------------------------------------------------------------------ latent attention with a latent of the queries
def _latent(shape, dtype, scale, eps, base, seed, own=True):
    H, dim, rot, vd, rank = shape
    q_rank = H * (dim + rot)
    rng = np.random.default_rng(seed)
    cols = q_rank + H * vd + rank + rot
    eye = np.eye(cols)
    bf = lambda a: _rounded(a, torch.bfloat16).numpy()  # noqa: E731
    tensors = {
        "dq": eye[:q_rank], "dq.norm": bf(1.0 + 0.2 * rng.standard_normal(q_rank)), "uq": np.eye(q_rank),
        "uk": bf(rng.standard_normal((H * dim, rank)) / np.sqrt(rank)), "uv": bf(rng.standard_normal((H * vd, rank)) / np.sqrt(rank)),
        "g": eye[q_rank : q_rank + H * vd], "o": np.zeros((cols, H * vd)),
    }
    if own:
        tensors.update({"dkv": eye[q_rank + H * vd :], "dkv.norm": bf(1.0 + 0.2 * rng.standard_normal(rank))})
    from rusty_llama_b200.spec import PartSpec

    params = {"hidden_size": cols, "num_heads": H, "dim": dim, "rot_dim": rot, "vdim": vd, "q_rank": q_rank, "kv_rank": rank, "scale": scale, "eps": eps,
              "sink": False, "gate": True, "own_kv": own, "window": 0,
              "position": PartSpec("rotary", {"rotary_dim": rot, "theta": base, "scaling": None, "interleaved": False}) if rot else PartSpec("none")}
    mix = {"heads": H, "dim": dim, "rot_dim": rot, "vdim": vd, "kv_rank": rank, "scale": scale, "rot": {"base": base, "dims": rot}}
    return params, tensors, {k: torch.as_tensor(v) for k, v in tensors.items()}, mix


LATENT_SHAPES = [(3, 12, 8, 20, 24), (4, 32, 16, 48, 64), (2, 64, 32, 64, 128), (5, 24, 16, 40, 96), (20, 8, 0, 16, 64)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", LATENT_SHAPES)
def test_one_latent_among_hundreds_and_a_reader_of_the_same_latents(shape, dtype):
    """One position's latent fits the later queries; it lies at page borders and far back.  A second mixer with other heads' maps reads the
    same latents without writing any."""
    from rusty_llama_b200.parts import MIXERS
    from rusty_llama_b200.spec import PartSpec

    H, dim, rot, vd, rank = shape
    eps, base, L = 1e-5, 1000.0, 330
    for target in (63, 64, 5):
        scale = 2.5 / np.sqrt(max(dim, 8))
        params, tensors, W, mix = _latent(shape, dtype, scale, eps, base, seed=target)
        mixer = MixerAlone("latent_attention", params, tensors, dtype)
        rp, rt, RW, rmix = _latent((H, dim, rot, vd, rank), dtype, scale, eps, base, seed=target + 1, own=False)
        reader = MIXERS.build(PartSpec("latent_attention", rp, "m."), mixer.rt)
        mixer.load(reader, rt)
        rng = np.random.default_rng(target + H)
        x = rng.standard_normal((L, W["dq"].shape[1]))
        n_q, n_kv = W["dq"].shape[0], x.shape[1] - rank - rot
        unit = rng.standard_normal(rank)
        x[target, n_kv : n_kv + rank] = 3.0 * unit
        fit = (W["uk"].view(H, dim, rank) @ torch.as_tensor(unit)).numpy()  # [H, dim]: the unrotated queries that this latent fits
        qv = x[:, :n_q].reshape(L, H, dim + rot)
        qv[target:, :, :dim] = 0.3 * qv[target:, :, :dim] + 3.0 * fit / np.sqrt((fit ** 2).mean())
        x = _rounded(x, dtype)
        rows = pf.latent_rows(x, W, "", mix, eps)
        ref = [_latent_plain(x, W, mix, eps, rows), _latent_plain(x, RW, rmix, eps, rows)]
        s = mixer.cache.open_sequence()
        got, at = [[], []], 0
        for n in [100, 2, 62, 130] + [1] * (L - 294):
            for g, o in zip(got, mixer.step([s], [x[at : at + n].numpy()], readers=[reader])):
                g.append(o[0])
            at += n
        mixer.cache.close_sequence(s)
        for who, g, r in zip(("own", "reader"), got, ref):
            g = torch.cat(g)
            tol = 3e-5 if dtype == torch.float32 else 4e-2
            assert float((g - r).abs().max()) <= tol * float(r.abs().max()), f"{who}, target {target}: row {int((g - r).abs().max(1).values.argmax())}"
        qn, qr = pf.latent_queries(x, W, "", mix, eps)
        score = (torch.einsum("hd,jhd->hj", qn[-1], (rows[0] @ W["uk"].T).view(L, H, dim)) + qr[-1] @ rows[1].T) * scale
        assert float(torch.softmax(score, dim=1)[:, target].max()) > 0.6  # the far latent holds most of a head's weight


def _latent_plain(x, W, mix, eps, rows):
    """What goes into the output projection: the plain mixer with an identity in its place."""
    return pf.latent_attention_mixer(x, dict(W, o=torch.eye(mix["heads"] * mix["vdim"], dtype=F64)), "", mix, eps, rows)


@pytest.mark.parametrize("interleaved", [False, True])
def test_pairs_of_the_shared_key_part(interleaved):
    """Rotated numbers beyond the pairs pass unchanged, in both layouts."""
    from rusty_llama_b200.kernels import ops

    T, rank, rot, pairs = 5, 8, 10, 3
    rng = np.random.default_rng(2)
    kv = rng.standard_normal((T, rank + rot))
    pages = torch.zeros((1, 1, 64, rank + rot), dtype=torch.float32, device="cuda")
    f = 0.4 ** np.arange(pairs)
    ops.latent_prep(None, _dev(kv, torch.float32), _dev(np.ones(rank), torch.float32), 1e-6, _dev(f, torch.float32), pairs, 1.0, _i32(np.arange(T)), _i32(np.zeros(T)),
                    _i32([[0]]), pages, None, 1, 0, rot, rank, interleaved)
    got = pages[0, 0, :T, rank:].to(F64).cpu().numpy()
    want = kv[:, rank:].copy()
    for i in range(pairs):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + pairs)
        c, s = np.cos(np.arange(T) * f[i]), np.sin(np.arange(T) * f[i])
        want[:, a], want[:, b] = kv[:, rank + a] * c - kv[:, rank + b] * s, kv[:, rank + b] * c + kv[:, rank + a] * s
    assert np.abs(got - want).max() < 1e-5


# ------------------------------------------------------------------ state-space layer
def _ssm(shape, dtype, eps, norm_groups, taps, a_log, dt_bias, seed):
    H, G, N, vd = shape
    inner, channels = H * vd, H * vd + 2 * G * N
    cols = inner + channels + H
    rng = np.random.default_rng(seed)
    bf = lambda a: _rounded(a, torch.bfloat16).numpy()  # noqa: E731
    tensors = {"in": np.eye(cols), "conv": bf(0.5 * rng.standard_normal((channels, taps))), "conv.b": bf(0.3 * rng.standard_normal(channels)),
               "dt_bias": bf(np.full(H, dt_bias) + 0.3 * rng.standard_normal(H)), "A_log": bf(np.full(H, a_log) + 0.5 * rng.standard_normal(H)),
               "D": bf(rng.standard_normal(H)), "norm": bf(1.0 + 0.3 * rng.standard_normal(inner)), "o": np.zeros((cols, inner))}
    params = {"hidden_size": cols, "num_heads": H, "vdim": vd, "state": N, "groups": G, "taps": taps, "norm_groups": norm_groups, "eps": eps}
    mix = {"heads": H, "vdim": vd, "state": N, "groups": G, "norm_groups": norm_groups}
    return params, tensors, {k: torch.as_tensor(v) for k, v in tensors.items()}, mix


def _ssm_plain(x, W, mix, eps, dtype):
    """The plain mixer before its output projection, with what the convolution's activation leaves rounded to the run's type, where
    the library stores it (a recurrence's sums cancel; its tolerance is then that of the kernels after it)."""
    H, vd, N, G = mix["heads"], mix["vdim"], mix["state"], mix["groups"]
    n, T = H * vd, x.shape[0]
    xbc = _rounded(pf.silu(pf.short_convolution(x[:, n : 2 * n + 2 * G * N], W["conv"], W["conv.b"])), dtype)
    y = pf.ssm_recurrence(xbc[:, :n].view(T, H, vd), xbc[:, n : n + G * N].view(T, G, N), xbc[:, n + G * N :].view(T, G, N),
                          pf.softplus(x[:, 2 * n + 2 * G * N :] + W["dt_bias"]), W["A_log"], W["D"])
    out = pf.gate_then_norm(y.reshape(T, n), x[:, :n], W["norm"], mix["norm_groups"], eps)
    if dtype == torch.float32:
        whole = pf.mamba2_mixer(x, dict(W, o=torch.eye(n, dtype=F64), **{"in": torch.eye(x.shape[1], dtype=F64)}), "", mix, eps)
        assert float((out - whole).abs().max()) <= 1e-5 * float(whole.abs().max())
    return out


SSM_SHAPES = [(3, 1, 24, 20, 5), (4, 2, 32, 32, 2), (4, 2, 128, 64, 4), (2, 1, 40, 100, 1), (6, 3, 48, 40, 2), (2, 2, 160, 24, 3)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", SSM_SHAPES)
def test_state_space_layer_in_portions(shape, dtype):
    """Slow, middling and fast forgetting; as one prompt (chunks), in portions with a ragged last chunk and down to two tokens, one by one."""
    H, G, N, vd, ng = shape
    L, eps = 203, 1e-5
    for case, (a_log, dt_bias, taps) in enumerate([(-6.0, -2.0, 4), (-1.0, 0.0, 3), (2.5, 1.0, 1)]):
        params, tensors, W, mix = _ssm(shape[:4], dtype, eps, ng, taps, a_log, dt_bias, seed=case)
        mixer = MixerAlone("mamba2", params, tensors, dtype, max_seqs=2)
        x = _rounded(np.random.default_rng(N + case).standard_normal((L, W["in"].shape[1])), dtype)
        ref = _ssm_plain(x, W, mix, eps, dtype)
        tol = 3e-5 if dtype == torch.float32 else 1.5e-2
        whole = mixer.run(x.numpy(), [L])
        assert float((whole - ref).abs().max()) <= tol * float(ref.abs().max()), f"case {case}: {float((whole - ref).abs().max() / ref.abs().max()):.2e} at row {int((whole - ref).abs().max(1).values.argmax())}"
        for cuts in ([64, 64, 64], [2, 2, 33, 65, 2, 40], [], [130]):
            got = mixer.run(x.numpy(), cuts)  # (the same slot again: its records read zero)
            assert float((got - ref).abs().max()) <= tol * float(ref.abs().max()), f"case {case}, cuts {cuts}: row {int((got - ref).abs().max(1).values.argmax())}"
            if dtype == torch.float32:
                assert torch.equal(got, whole), f"case {case}, cuts {cuts}: other bits"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("form", ["chunked", "token by token"])
def test_what_is_written_once_is_read_far_away(form, dtype):
    """Only token 3 has a key in direction 0 and the state never forgets: a query in that direction reads exactly dt x_3 at every chunk's
    first and last token, and nothing before it."""
    from rusty_llama_b200.kernels import ops

    if form == "chunked" and dtype == torch.float32:
        pytest.skip("prompts of 32-bit runs go token by token")
    H, G, N, vd, T = 4, 2, 48, 40, 260
    rng = np.random.default_rng(4)
    rows = np.zeros((T, H * vd + 2 * G * N))
    rows[:, : H * vd] = rng.standard_normal((T, H * vd))
    rows[:, H * vd :] = 0.3 * rng.standard_normal((T, 2 * G * N))
    B, C = rows[:, H * vd : H * vd + G * N].reshape(T, G, N), rows[:, H * vd + G * N :].reshape(T, G, N)
    B[:, :, 0], B[3, :, 0] = 0.0, 2.0
    reads = [2, 3, 63, 64, 127, 128, 191, 192, 255, 259]
    C[reads] = 0.0
    C[reads, :, 0] = 1.0
    x = _dev(rows, dtype)
    xv, Bv, Cv = x[:, : H * vd], x[:, H * vd : H * vd + G * N], x[:, H * vd + G * N :]
    log_a, dt = torch.zeros((T, H), device="cuda"), torch.full((T, H), 0.5, device="cuda")
    state = torch.zeros((3, H, N, vd), device="cuda")
    args = (Cv, Bv, xv, log_a, dt, state, _i32([2]), _i32([0, T]), H, N, vd)
    if form == "chunked":
        scratch = torch.full((ops.scalar_decay_chunked_scratch_floats(1, T, H, N, vd),), float("nan"), device="cuda")
        y = ops.scalar_decay_chunked(*args, T, scratch, qk_heads=G)
    else:
        y = ops.gated_attn(*args, qk_heads=G)
    want = rows[3, : H * vd] if dtype == torch.float32 else _rounded(rows[3, : H * vd], dtype).numpy()
    for t in reads:
        got = y[t].to(F64).cpu().numpy()
        assert np.abs(got - (want if t >= 3 else 0.0)).max() <= 1e-4 * np.abs(want).max(), t
    assert float(state[:2].abs().sum()) == 0.0 and bool(torch.isfinite(y).all())


def test_chunked_recurrence_against_token_by_token_with_strong_decays():
    """Decay sums in the thousands inside a chunk, two sequences of unequal lengths, slots out of order, states that are not zero."""
    from rusty_llama_b200.kernels import ops

    rng = np.random.default_rng(9)
    for H, G, N, vd in ((4, 2, 128, 64), (2, 1, 33, 17), (3, 3, 64, 128), (2, 2, 16, 16)):
        lens = (131, 64, 1)
        T = sum(lens)
        cols = H * vd + 2 * G * N + 3
        x = _dev(rng.standard_normal((T, cols)), torch.bfloat16)
        v, k, q = x[:, : H * vd], x[:, H * vd : H * vd + G * N], x[:, H * vd + G * N : H * vd + 2 * G * N]
        for strength in (0.001, 0.3, 60.0):
            log_a = -strength * _dev(rng.uniform(0.1, 1.0, (T, H)), torch.float32)
            dt = _dev(rng.uniform(0.1, 2.0, (T, H)), torch.float32)
            st = _dev(rng.standard_normal((5, H, N, vd)), torch.float32)
            args = (q, k, v, log_a, dt)
            tail = (_i32([4, 0, 2]), _i32(np.concatenate([[0], np.cumsum(lens)])), H, N, vd)
            s1, s2 = st.clone(), st.clone()
            a = ops.gated_attn(*args, s1, *tail, qk_heads=G)
            scratch = torch.full((ops.scalar_decay_chunked_scratch_floats(3, max(lens), H, N, vd),), float("nan"), device="cuda")
            b = ops.scalar_decay_chunked(*args, s2, *tail, max(lens), scratch, qk_heads=G)
            assert float((a - b).abs().max()) <= 1e-3 * float(a.abs().max()), (H, strength, float((a - b).abs().max() / a.abs().max()))
            assert float((s1 - s2).abs().max()) <= 1e-4 * float(s1.abs().max()) and torch.equal(s2[[1, 3]], st[[1, 3]])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 4, 9])
def test_single_tokens_through_the_convolution_with_a_bias(dtype, taps):
    """The kernel for single tokens makes the same bits as the one for portions, and leaves the same record."""
    from rusty_llama_b200.kernels import ops

    rng = np.random.default_rng(taps)
    C, S = 43, 3
    w, b = _dev(rng.standard_normal((taps, C)), torch.float32), _dev(rng.standard_normal(C), torch.float32)
    state = _dev(rng.standard_normal((5, max(taps - 1, 1), C)), torch.float32)[:, : taps - 1].contiguous() if taps > 1 else None
    x = _dev(rng.standard_normal((S, C + 5)), dtype)[:, :C]
    slots, start, seq = _i32([4, 0, 2]), _i32([0, 1, 2, 3]), _i32([0, 1, 2])
    one, two = (None if state is None else state.clone() for _ in range(2))
    y1 = ops.short_conv(x, w, one, slots, start, seq, bias=b, single=True)
    y2 = ops.short_conv(x, w, two, slots, start, seq, bias=b)
    assert torch.equal(y1, y2)
    if state is not None:
        assert torch.equal(one, two) and torch.equal(one[[1, 3]], state[[1, 3]]) and torch.equal(one[[4, 0, 2], -1], x.float())
    for i, slot in enumerate([4, 0, 2]):
        before = np.zeros((0, C)) if state is None else state[slot].to(F64).cpu().numpy()
        seen = torch.as_tensor(np.concatenate([before, x[i : i + 1].to(F64).cpu().numpy()]))
        want = pf.silu(pf.short_convolution(seen, w.to(F64).cpu().T, b.to(F64).cpu())[-1])
        assert float((y1[i].to(F64).cpu() - want).abs().max()) <= (2e-6 if dtype == torch.float32 else 8e-3) * max(1.0, float(want.abs().max()))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(60, 3, 5), (128, 4, 4), (4096, 64, 8), (68, 2, 1), (10240, 80, 2)])
def test_gate_before_the_norm(sizes, dtype):
    from rusty_llama_b200.kernels import ops

    n, H, groups = sizes
    rng = np.random.default_rng(n)
    T = 70
    y = rng.standard_normal((T, n)) * (10.0 ** (np.arange(n) * groups // n % 3))  # parts of a row that differ by factors of ten
    x, z = _rounded(rng.standard_normal((T, n)), dtype), _rounded(2.0 * rng.standard_normal((T, n)), dtype)
    D, w = rng.standard_normal(H), rng.standard_normal(n)
    want = pf.gate_then_norm(torch.as_tensor(y) + torch.as_tensor(np.repeat(D, n // H)) * x, z, torch.as_tensor(w), groups, 1e-6)
    args = [_dev(a, torch.float32) for a in (y, D, w)]
    got = ops.ssm_gate_norm(args[0], _dev(x, dtype), args[1], _dev(z, dtype), args[2], 1e-6, groups, dtype)
    tol = 5e-6 if dtype == torch.float32 else 8e-3
    assert float((got.to(F64).cpu() - want).abs().max()) <= tol * float(want.abs().max())
    few = ops.ssm_gate_norm(args[0][:3], _dev(x[:3], dtype), args[1], _dev(z[:3], dtype), args[2], 1e-6, groups, dtype)
    assert torch.equal(few, got[:3])  # a row's bits do not depend on how many rows there are


# ------------------------------------------------------------------ gated residual, norm in groups, logits
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(96, 3), (68, 1), (100, 20), (2048, 8), (4096, 1), (7680, 5), (66, 11)])
def test_gated_result_and_norm_in_groups(sizes, dtype):
    """The sum, the gate and the norm in one kernel: one part and several, with and without a gate, all rows and some, and the sum alone."""
    from rusty_llama_b200.kernels import ops

    d, groups = sizes
    rng = np.random.default_rng(d)
    for T, parts in ((3, 1), (80, 1), (5, 3), (70, 2)):
        x = rng.standard_normal((T, d)) * 10.0 ** (np.arange(d) * groups // d % 3)
        x = _rounded(x, torch.float32)
        delta = _rounded(rng.standard_normal((parts, T, d)), torch.float32 if parts > 1 else dtype)
        z, b, w = _rounded(2.0 * rng.standard_normal((T, d)), dtype), _rounded(rng.standard_normal(d), torch.float32), _rounded(rng.standard_normal(d), torch.float32)
        dd = _dev(delta, torch.float32) if parts > 1 else _dev(delta[0], dtype)
        zrows = torch.zeros((T, d + 8), dtype=dtype, device="cuda")
        zrows[:, :d] = _dev(z, dtype)
        gate = (zrows[:, :d], _dev(b, torch.float32))
        tol = 5e-6 if dtype == torch.float32 else 8e-3
        for use_gate in (True, False):
            summed = x + delta.sum(0) * (pf.logistic(z + b) if use_gate else 1.0)
            want = pf.grouped_norm(summed, w, groups, 1e-5)
            xs = _dev(x, torch.float32)
            got = ops.gated_add_rmsnorm(xs, dd, gate if use_gate else None, _dev(w, torch.float32), 1e-5, groups, dtype)
            assert float((xs.to(F64).cpu() - summed).abs().max()) <= 1e-6 * float(summed.abs().max())
            assert float((got.to(F64).cpu() - want).abs().max()) <= tol * float(want.abs().max())
            rows = [T - 1, 0]
            xr = _dev(x, torch.float32)
            some = ops.gated_add_rmsnorm(xr, dd, gate if use_gate else None, _dev(w, torch.float32), 1e-5, groups, dtype, rows=_i32(rows), write_x=False)
            assert torch.equal(some, got[rows]) and torch.equal(xr, _dev(x, torch.float32))
            alone = _dev(x, torch.float32)
            assert ops.gated_add_rmsnorm(alone, dd, gate if use_gate else None, None, 0.0, 1, dtype) is None and torch.equal(alone, xs)
        first = ops.gated_add_rmsnorm(_dev(x, torch.float32), None, None, _dev(w, torch.float32), 1e-5, groups, dtype)
        want = pf.grouped_norm(x, w, groups, 1e-5)
        assert float((first.to(F64).cpu() - want).abs().max()) <= tol * float(want.abs().max())


def test_logits_scale_and_cap():
    from rusty_llama_b200.kernels import ops

    z = np.random.default_rng(1).standard_normal((7, 1003)) * 30
    for scale, cap in ((2.0, 15.0), (0.5, 0.0), (1.0, 3.0)):
        y = _dev(z, torch.float32)
        want = pf.cap_logits(y.to(F64).cpu(), scale, cap)
        assert ops.scale_softcap(y, scale, cap) is y
        assert float((y.to(F64).cpu() - want).abs().max()) <= 3e-6 * float(want.abs().max())


def test_what_a_block_leaves_pending_is_gated_before_it_is_added():
    from rusty_llama_b200.parts.base import ResidualStream

    rng = np.random.default_rng(3)
    x, delta, z, b = (rng.standard_normal(s) for s in ((4, 96), (4, 96), (4, 96), (96,)))
    stream = ResidualStream(_dev(x, torch.float32), torch.float32)
    stream.add(_dev(delta, torch.float32), gate=(_dev(z, torch.float32), _dev(b, torch.float32)))
    stream.add(_dev(delta, torch.float32))  # flushes the first
    stream.flush()
    want = torch.as_tensor(x) + torch.as_tensor(delta) * (1.0 + pf.logistic(torch.as_tensor(z + b)))
    assert stream.pending is None and stream.pending_gate is None
    assert float((stream.x.to(F64).cpu() - want).abs().max()) < 1e-5


@pytest.mark.parametrize("dtype", DTYPES)
def test_experts_weighted_over_the_chosen_ones(dtype):
    from rusty_llama_b200.kernels import ops

    rng = np.random.default_rng(6)
    T, d, E, top = 40, 64, 7, 3
    h, w = _rounded(rng.standard_normal((T, d)), dtype), _rounded(rng.standard_normal((E, d)), torch.float32)
    ids, weights, _ = ops.moe_router(_dev(h, dtype), _dev(w, torch.float32), None, E, top, True)
    chosen, want = pf.route(h, {"r.router": w}, "r.", top)
    assert torch.equal(ids.cpu().to(torch.long), chosen)
    assert float((weights.to(F64).cpu() - want).abs().max()) <= 1e-5
