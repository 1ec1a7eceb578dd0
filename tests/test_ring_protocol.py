"""The ring protocol of the TMA / tensor-core kernels (csrc/gemm_tc.cu and its relatives), checked as a model on
the CPU: every interleaving of the four actors on a small ring.

    producer     requests slice i into stage i % S once the stage's `empty` barrier shows that the products of
                 slice i - S are done (no wait for the first S slices); the parity it waits on starts at 1 and flips
                 at every wrap of the ring
    copy engine  lands the requested slices in any order; a landed slice completes one phase of its stage's
                 `full` barrier
    issuer       waits for slice i's stage on `full` (parity (i / S) & 1) and issues its products; optionally it asks
                 about the NEXT stage at the same moment and skips the next wait after a yes
    tensor pipe  finishes issued slices in order; a finished slice completes one phase of its stage's `empty` barrier

A barrier is modelled as its number of completed phases, and a wait on parity P succeeds iff the barrier's current
phase has the other parity (`mbarrier.try_wait.parity` / `test_wait.parity`).  Checked: no slice's products are issued
before its data has landed, and nothing ever waits for ever.  (The kernels' arithmetic for stage and parity is
restated here, not imported: a change there has to be made here too, and then checked again.)"""

from collections import deque

import pytest


def _ok(completed: int, parity: int) -> bool:
    return (completed & 1) != parity


def _explore(S: int, T: int, ask_ahead: bool):
    """Breadth-first over all reachable states; returns (states visited, first problem found or None)."""
    start = (0, (), (0,) * S, (0,) * S, 0, 0, (), frozenset())
    seen, queue = {start}, deque([start])
    while queue:
        p_it, flying, full, empty, i_it, ready, issued, landed = st = queue.popleft()
        nxt = []
        if p_it < T:  # producer
            s, parity = p_it % S, ((p_it // S) & 1) ^ 1
            if p_it < S or _ok(empty[s], parity):
                nxt.append((p_it + 1, flying + (p_it,), full, empty, i_it, ready, issued, landed))
        for k, sl in enumerate(flying):  # copy engine
            f = list(full)
            f[sl % S] += 1
            nxt.append((p_it, flying[:k] + flying[k + 1:], tuple(f), empty, i_it, ready, issued, landed | {sl}))
        if i_it < T:  # issuer
            s, parity = i_it % S, (i_it // S) & 1
            if ready or _ok(full[s], parity):
                if i_it not in landed:
                    return len(seen), f"slice {i_it} issued before its data landed"
                yes = 0
                if ask_ahead:
                    s1, parity1 = (i_it + 1) % S, ((i_it + 1) // S) & 1
                    yes = 1 if _ok(full[s1], parity1) else 0
                nxt.append((p_it, flying, full, empty, i_it + 1, yes, issued + (i_it,), landed))
        if issued:  # tensor pipe
            e = list(empty)
            e[issued[0] % S] += 1
            nxt.append((p_it, flying, full, tuple(e), i_it, ready, issued[1:], landed))
        if not nxt and (p_it < T or i_it < T):
            return len(seen), f"nothing can move at producer {p_it}, issuer {i_it}"
        for n in nxt:
            if n not in seen:
                seen.add(n)
                queue.append(n)
    return len(seen), None


@pytest.mark.parametrize("S, T", [(2, 7), (3, 10), (4, 11), (5, 12)])
@pytest.mark.parametrize("ask_ahead", [False, True])
def test_ring_of_stages_never_issues_early_and_never_stalls(S, T, ask_ahead):
    states, problem = _explore(S, T, ask_ahead)
    assert problem is None, problem
    assert states > T * S


def test_the_model_sees_a_wrong_parity():
    """The checker itself: an issuer that waits on the producer's parity convention is caught."""
    S, T = 3, 8
    # the same exploration with the issuer's parity flipped
    start = (0, (), (0,) * S, 0, frozenset())
    seen, queue, problem = {start}, deque([start]), None
    while queue and problem is None:
        p_it, flying, full, i_it, landed = queue.popleft()
        nxt = []
        if p_it < min(T, S):
            nxt.append((p_it + 1, flying + (p_it,), full, i_it, landed))
        for k, sl in enumerate(flying):
            f = list(full)
            f[sl % S] += 1
            nxt.append((p_it, flying[:k] + flying[k + 1:], tuple(f), i_it, landed | {sl}))
        if i_it < S and _ok(full[i_it % S], ((i_it // S) & 1) ^ 1):  # wrong: succeeds on a fresh barrier
            if i_it not in landed:
                problem = f"slice {i_it} issued before its data landed"
            nxt.append((p_it, flying, full, i_it + 1, landed))
        for n in nxt:
            if n not in seen:
                seen.add(n)
                queue.append(n)
    assert problem is not None


def _explore_attention(T: int, p_barriers: int):
    """csrc/attention_prefill_tc.cu over T key tiles, with `p_barriers` barriers for "the probabilities are ready".  Actors: the
    producer (K and V tiles into two stages each; a K stage is free when the S it fed is complete, a V stage when its P V is), the
    copy engine, the issuer (S 0, S 1, then for every tile j: wait for P j and V j, issue P V j, wait for K j + 2, issue S j + 2),
    the tensor pipe (in order), and the softmax warps as one actor (wait for S j, announce P j).  Returns the first problem
    found or None."""
    loads = [(kind, j) for j in range(T) for kind in "KV"]
    order = [("S", j) for j in range(min(2, T))]
    for j in range(T):
        order.append(("O", j))
        if j + 2 < T:
            order.append(("S", j + 2))
    zero = (0, 0)
    bump = lambda b, i: tuple(n + (k == i) for k, n in enumerate(b))  # noqa: E731
    # producer's place, copies in flight, completed phases of k_full, v_full, s_full, pv_done, p_ready, issuer's place, half a wait, issued, softmax's place
    start = (0, (), zero, zero, zero, zero, (0,) * p_barriers, 0, 0, (), 0)
    seen, queue = {start}, deque([start])
    while queue:
        lo, fly, kf, vf, sf, pv, pr, io, half, iss, sm = queue.popleft()
        nxt = []
        if lo < len(loads):
            kind, j = loads[lo]
            if j < 2 or _ok((sf if kind == "K" else pv)[j & 1], ((j >> 1) - 1) & 1):
                nxt.append((lo + 1, fly + (loads[lo],), kf, vf, sf, pv, pr, io, half, iss, sm))
        for n, (kind, j) in enumerate(fly):
            k2, v2 = (bump(kf, j & 1), vf) if kind == "K" else (kf, bump(vf, j & 1))
            nxt.append((lo, fly[:n] + fly[n + 1:], k2, v2, sf, pv, pr, io, half, iss, sm))
        if io < len(order):
            kind, j = order[io]
            if kind == "S":
                if _ok(kf[j & 1], (j >> 1) & 1):
                    nxt.append((lo, fly, kf, vf, sf, pv, pr, io + 1, 0, iss + (order[io],), sm))
            elif half == 0:
                if _ok(pr[j % p_barriers], (j // p_barriers) & 1):
                    if sm <= j:
                        return f"P V {j} goes on before its probabilities are there"
                    nxt.append((lo, fly, kf, vf, sf, pv, pr, io, 1, iss, sm))
            elif _ok(vf[j & 1], (j >> 1) & 1):
                nxt.append((lo, fly, kf, vf, sf, pv, pr, io + 1, 0, iss + (order[io],), sm))
        if iss:
            kind, j = iss[0]
            s2, o2 = (bump(sf, j & 1), pv) if kind == "S" else (sf, bump(pv, j & 1))
            nxt.append((lo, fly, kf, vf, s2, o2, pr, io, half, iss[1:], sm))
        if sm < T and _ok(sf[sm & 1], (sm >> 1) & 1):
            nxt.append((lo, fly, kf, vf, sf, pv, bump(pr, sm % p_barriers), io, half, iss, sm + 1))
        if not nxt and (lo < len(loads) or io < len(order) or sm < T):
            return f"nothing can move: producer at {loads[lo:lo + 1]}, issuer at {order[io:io + 1]}, softmax at {sm}"
        for n in nxt:
            if n not in seen:
                seen.add(n)
                queue.append(n)
    return None


@pytest.mark.parametrize("T", [1, 2, 3, 4, 5, 8])
def test_prompt_attention_never_stalls_with_a_barrier_per_score_buffer(T):
    assert _explore_attention(T, p_barriers=2) is None


def test_prompt_attention_with_one_barrier_for_the_probabilities_can_stall():
    """Tile j + 1's scores are under way before the issuer looks for tile j's probabilities, so the softmax warps can announce both
    first; the parity of a single barrier is then back where it was, and the producer ends waiting for a value stage."""
    problem = _explore_attention(4, p_barriers=1)
    assert problem is not None and "nothing can move" in problem and "('V'" in problem
