"""Nugopel on the GPU against the plain implementation (tests/plain_nugopel.py).

Mechanisms alone (parts and kernels against the plain function of the same
mechanism): latent attention without positions on an own latent and on another
layer's, its channel gates in the value product; windowed attention after norms
over whole projections and a rotation of halves, with one added to the
softmax's denominator, on the every-size and the tensor-core kernels; both over
pages of which those that nothing may see are poisoned, in prompts, portions
and decoding at lengths around page and window borders; one key made to stand
out far away, just inside and just outside the window; the share the added one
takes; the rotation at large positions; the mixture of experts; norms stored
less one.  Then whole models of five configurations, in 32-bit and bfloat16:
whole prompts, prefill against token-by-token decoding, portions down to two
tokens, batches of unequal requests in a pool so small that pages and slots are
used again, long decoding from the first token, the stream after every layer,
and greedy generation through the engine and the programs."""
import json
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_nugopel as plain
import replay
import tiny_nugopel as tiny
from gpu_util import assert_close, dev, rounded

pytestmark = pytest.mark.gpu

F32, BF16 = torch.float32, torch.bfloat16
# Largest |engine - plain| on logits, times max(1, max|plain|): fp32 sums against float64; bfloat16 rounds
# activations and cache rows to 8 bits of mantissa.
TOL = {"float32": 3e-5, "bfloat16": 9e-2}
KERNEL_TOL = {F32: 2e-5, BF16: 3e-2}


class Owed:
    """What a product leaves when its reader is to add its split sums up: planes [splits, rows, columns] and a bias."""

    def __init__(self, sums, bias=None):
        self.sums, self.splits, self.bias = sums, sums.shape[0], bias


# ---------------------------------------------------------------------------------------------------
# mixers: the parts themselves over a paged cache, with weights that pick queries, keys, latents and gates out of the
# input, so that a test can make them what it wants
# ---------------------------------------------------------------------------------------------------
class Paged:
    """Requests of given lengths over one paged cache with block tables in random order."""

    group, page_size = 0, 0

    def __init__(self, rng, lengths, page, k_shape, v_shape=None, dtype=F32, window=None):
        self.lengths, self.page_size, self.window = lengths, page, window
        blocks = [-(-n // page) for n in lengths]
        order = rng.permutation(sum(blocks) + 3)
        self.table = np.full((len(lengths), max(blocks) + 1), -1, dtype=np.int32)
        at = 0
        for r, b in enumerate(blocks):
            self.table[r, :b] = order[at : at + b]
            at += b
        slots = (sum(blocks) + 3) * page
        self.k = torch.empty((slots, *k_shape), dtype=dtype, device="cuda")
        self.v = torch.empty((slots, *v_shape), dtype=dtype, device="cuda") if v_shape else None
        self.clear()

    def clear(self):
        self.k.fill_(60.0)  # what lies in slots that nothing may see must not matter
        if self.v is not None:
            self.v.fill_(-900.0)

    def poison_passed_pages(self, spans):
        """What the cache manager may have given away by the next step: pages behind the window."""
        for r, _, hi in spans if self.window else ():
            for b in range(max(0, hi - self.window + 1) // self.page_size):
                s = self.table[r, b] * self.page_size
                self.k[s : s + self.page_size] = 60.0
                self.v[s : s + self.page_size] = -900.0


class Group:
    pass


class Step:
    """What a mixer reads of a step's context, for the rows ``spans`` = [(request, lo, hi)]."""

    capturing = False

    def __init__(self, case, spans):
        counts = [hi - lo for _, lo, hi in spans]
        self.n_tokens, self.n_seqs, self.max_q_len = sum(counts), len(spans), max(counts)
        self.decode_only = self.max_q_len == 1
        self.fresh = not self.decode_only and all(lo == 0 for _, lo, _ in spans)
        self.max_kv_len = self.max_context = max(hi for _, _, hi in spans)
        self.positions = dev(np.concatenate([np.arange(lo, hi, dtype=np.int32) for _, lo, hi in spans]))
        self.seq_of_token = dev(np.concatenate([np.full(c, s, dtype=np.int32) for s, c in enumerate(counts)]))
        self.q_start = dev(np.concatenate([[0], np.cumsum(counts)]).astype(np.int32))
        self.kv_len = dev(np.array([hi for _, _, hi in spans], dtype=np.int32))
        self.status = torch.zeros(4, dtype=torch.int32, device="cuda")
        g = Group()
        page = g.page_size = case.page_size
        g.block_table = dev(case.table[[r for r, _, _ in spans]])
        g.slot_map = dev(np.array([case.table[r, j // page] * page + j % page for r, lo, hi in spans for j in range(lo, hi)], dtype=np.int32))
        self.groups, self.first_values = [g], None

    @staticmethod
    def buf(shape, dtype):
        return torch.empty(shape, dtype=dtype, device="cuda")


def run_part(part, case, rows, spans, dtype, writes=True):
    ctx = Step(case, spans)
    x = dev(np.concatenate([rows[r][lo:hi] for r, lo, hi in spans]), dtype)
    h = torch.full((x.shape[0], part.hidden_out), 7.0, dtype=F32, device="cuda")
    owed = part.forward(ctx, x, h, case, writes, store=True)
    assert owed is None and int(ctx.status.sum()) == 0
    return h.cpu().numpy()


def in_steps(part, case, rows, dtype, cuts, reader=None):
    """Every request whole in one step; then again from an empty cache in portions of ``cuts`` (1: decoding) with all requests
    in every step.  ``reader``: a part that runs after ``part`` on the rows it cached; the results are then its."""
    def step(spans):
        out = run_part(part, case, rows, spans, dtype)
        return out if reader is None else run_part(reader, case, rows, spans, dtype, writes=False)

    whole = step([(r, 0, n) for r, n in enumerate(case.lengths)])
    split = np.cumsum([0] + list(case.lengths))
    out = [[whole[split[r] : split[r + 1]] for r in range(len(rows))]]
    case.clear()
    got, at, count = [[] for _ in rows], [0] * len(rows), 0
    while any(at[r] < n for r, n in enumerate(case.lengths)):
        spans = []
        for r, n in enumerate(case.lengths):
            if at[r] < n:
                spans.append((r, at[r], at[r] + min(cuts[(count + r) % len(cuts)], n - at[r])))
        count += 1
        res, k = step(spans), 0
        for r, lo, hi in spans:
            got[r].append(res[k : k + hi - lo])
            k += hi - lo
            at[r] = hi
        case.poison_passed_pages(spans)
    out.append([np.concatenate(g) for g in got])
    return out


def loaded(part, w, prefix, dtype, hidden_out):
    part.load({n: dev(v, dtype) for n, v in w.items() if n.startswith(prefix)})
    part.hidden_out = hidden_out
    return part


def latent_part(w, m, width, dtype, own, eps=1e-5, prefix="a."):
    from alofa_b200.config.spec import PartSpec
    from alofa_b200.parts.base import Runtime, build_part

    part = build_part("mixer", PartSpec("latent_attention", {"hidden_size": width, "heads": m["heads"], "dim": m["dim"], "rot_dim": 0, "vdim": m["vdim"], "kv_rank": m["kv_rank"],
                                                              "q_rank": 0, "scale": m["scale"], "eps": eps, "gate": "channel", "own_latent": own}, prefix=prefix),
                      Runtime(torch.device("cuda"), dtype))
    return loaded(part, w, prefix, dtype, m["heads"] * m["vdim"])


def latent_weights(rng, m, dtype, prefix="a.", own=True, columns=None):
    """The input is [q | latent before its norm | gate logits]; the projections pick their columns; the output projection is the identity."""
    H, d, dv, r = m["heads"], m["dim"], m["vdim"], m["kv_rank"]
    q0, c0, g0, width = columns or (0, H * d, H * d + r, H * d + r + H * dv)
    eye = np.eye(width)
    w = {"q": eye[q0 : q0 + H * d], "uk": rounded(rng.standard_normal((H * d, r)) / np.sqrt(r), dtype), "uv": rounded(rng.standard_normal((H * dv, r)) / np.sqrt(r), dtype),
         "g": eye[g0 : g0 + H * dv], "o": np.eye(H * dv)}
    if own:
        w.update({"dkv": eye[c0 : c0 + r], "dkv.norm": rounded(1 + 0.3 * rng.standard_normal(r), dtype)})
    return {prefix + n: v for n, v in w.items()}, width


def latent_mixer(H, d, dv, r, scale=None):
    return {"heads": H, "dim": d, "vdim": dv, "kv_rank": r, "scale": scale or 2.0 / np.sqrt(d)}


LATENTS = [(F32, 5, 24, 20, 40, 16), (F32, 3, 10, 7, 33, 64), (F32, 18, 8, 10, 300, 16), (BF16, 5, 24, 20, 40, 16), (BF16, 4, 32, 48, 64, 64), (BF16, 20, 16, 24, 64, 16),
           (BF16, 6, 64, 32, 128, 48), (BF16, 2, 128, 64, 512, 64), (BF16, 70, 16, 16, 32, 64), (BF16, 1, 16, 8, 96, 32), (BF16, 3, 12, 5, 64, 64)]


@pytest.mark.parametrize("dtype,H,d,dv,r,page", LATENTS)
def test_latent_attention_on_its_own_latent_and_on_another_layers(dtype, H, d, dv, r, page):
    """Whole prompts, portions and decoding at lengths around pages; a second layer with other heads, sizes and gates on the
    rows the first one cached."""
    rng = np.random.default_rng(3)
    m, m2 = latent_mixer(H, d, dv, r), latent_mixer(H + 1, 16, 12, r)
    w, width = latent_weights(rng, m, dtype)
    n2 = m2["heads"] * 16 + m2["heads"] * 12  # the second layer's queries and gates stand in columns of their own
    w2, _ = latent_weights(rng, m2, dtype, "b.", False, (width, 0, width + m2["heads"] * 16, width + n2))
    w = {n: np.pad(v, ((0, 0), (0, n2))) if v.ndim == 2 and v.shape[1] == width else v for n, v in w.items()}
    lengths = sorted({1, 2, page - 1, page, page + 1, 31, 33, 130, 150 if dtype == F32 else 300})
    rows = [rounded(rng.standard_normal((n, width + n2)), dtype) for n in lengths]
    first = latent_part(w, m, width + n2, dtype, True)
    second = latent_part(w2, m2, width + n2, dtype, False, prefix="b.")
    latents = [plain.latent(w, "a.", x, 1e-5) for x in rows]
    for reader, ww, p, mm in ((None, w, "a.", m), (second, w2, "b.", m2)):
        want = [plain.latent_attention(ww, p, mm, x, c) for x, c in zip(rows, latents)]
        for cuts in ((1,), (5, 2, 16, 3, 2, 64)):
            case = Paged(rng, lengths, page, (r,), dtype=dtype)
            for what, got in zip(("whole", f"portions of {cuts}"), in_steps(first, case, rows, dtype, cuts, reader)):
                for i, n in enumerate(lengths):
                    assert_close(got[i], want[i], KERNEL_TOL[dtype], f"{what}: request of {n} tokens, own {reader is None}")


@pytest.mark.parametrize("H,d,dv,r,page", [(4, 32, 48, 64, 64), (3, 64, 64, 128, 16), (2, 128, 64, 40, 48), (16, 16, 16, 96, 64)])
@pytest.mark.parametrize("lengths", [[128], [130, 257, 192], [500, 1, 64, 63], [65, 300]])
def test_prompts_alone_attend_to_keys_and_values_made_from_their_latents(H, d, dv, r, page, lengths):
    """bfloat16 steps of prompts that all start in them, of whole pages and not, then a portion and single tokens over the same
    cache, which go the other way; a second layer on the same rows."""
    rng = np.random.default_rng(21)
    m, m2 = latent_mixer(H, d, dv, r), latent_mixer(H + 1, 32, 16, r)
    w, width = latent_weights(rng, m, BF16)
    n2 = (H + 1) * 48
    w2, _ = latent_weights(rng, m2, BF16, "b.", False, (width, 0, width + (H + 1) * 32, width + n2))
    w = {n: np.pad(v, ((0, 0), (0, n2))) if v.ndim == 2 and v.shape[1] == width else v for n, v in w.items()}
    rows = [rounded(rng.standard_normal((n + 6, width + n2)), BF16) for n in lengths]
    first, second = latent_part(w, m, width + n2, BF16, True), latent_part(w2, m2, width + n2, BF16, False, prefix="b.")
    assert first.tells_fresh and second.tells_fresh and not latent_part(w, m, width + n2, F32, True).tells_fresh
    case = Paged(rng, [n + 6 for n in lengths], page, (r,), dtype=BF16)
    latents = [plain.latent(w, "a.", x, 1e-5) for x in rows]
    want = [[plain.latent_attention(w, "a.", m, x, c) for x, c in zip(rows, latents)], [plain.latent_attention(w2, "b.", m2, x, c) for x, c in zip(rows, latents)]]
    calls = []
    for part in (first, second):
        part.attend_unfolded = lambda *a, f=part.attend_unfolded: calls.append(1) or f(*a)
    for lo, hi in ((0, 0), (0, 4), (4, 5), (5, 6)):  # the prompts; four tokens more of each; two single ones
        spans = [(i, n + lo if hi else 0, n + hi) for i, n in enumerate(lengths)]
        for part, ref, writes in ((first, want[0], True), (second, want[1], False)):
            got = run_part(part, case, rows, spans, BF16, writes)
            assert_close(got, np.concatenate([ref[i][a:b] for i, a, b in spans]), KERNEL_TOL[BF16], f"tokens {lo} to {hi}")
    assert len(calls) == 2, "the prompts alone should have gone over keys and values of their own"


@pytest.mark.parametrize("dtype,H,d,dv,r", [(F32, 2, 16, 8, 24), (BF16, 2, 16, 8, 24), (BF16, 4, 32, 16, 64), (BF16, 17, 16, 16, 64)])
def test_latent_attention_finds_one_far_key_among_hundreds(dtype, H, d, dv, r):
    """Key 3 of 700 matches the last query far better than any other: the output is its value times the gates."""
    rng = np.random.default_rng(5)
    m = latent_mixer(H, d, dv, r, scale=1.0)
    w, width = latent_weights(rng, m, dtype)
    w["a.dkv.norm"] = np.ones(r)
    w["a.uk"][:, 0] *= 3.0  # the latent's first number weighs most in the keys ...
    x = rounded(rng.standard_normal((700, width)), dtype)
    x[:, H * d] = 0.0
    x[3, H * d : H * d + r] = 9.0 * (np.arange(r) == 0)  # ... and key 3 alone has it
    k3 = plain.latent(w, "a.", x, 1e-5)[3] @ w["a.uk"].T
    x[699, : H * d] = 12.0 * k3 / np.sqrt((k3 * k3).reshape(H, d).sum(-1)).repeat(d) ** 2 * np.sqrt(d)
    x = rounded(x, dtype)
    c = plain.latent(w, "a.", x, 1e-5)
    want = plain.latent_attention(w, "a.", m, x, c)
    value = (c[3] @ w["a.uv"].T) * plain.sigmoid(x[699, -H * dv :])
    assert np.abs(want[699] - value).max() < 0.25 * np.abs(value).max(), "the test's far key does not stand out"
    case = Paged(rng, [700], 16, (r,), dtype=dtype)
    part = latent_part(w, m, width, dtype, True)
    run_part(part, case, [x], [(0, 0, 699)], dtype)
    assert_close(run_part(part, case, [x], [(0, 699, 700)], dtype), want[699:], KERNEL_TOL[dtype], "last query")


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("batches,m,n,k", [(3, 1, 24, 16), (5, 70, 33, 40), (2, 129, 64, 100), (4, 64, 7, 9)])
def test_gate_in_the_batched_product(dtype, batches, m, n, k):
    from alofa_b200.csrc import ops

    rng = np.random.default_rng(6)
    x, wt = rounded(rng.standard_normal((m, batches, k)), dtype), rounded(rng.standard_normal((batches, n, k)) / np.sqrt(k), dtype)
    gate = rounded(3 * rng.standard_normal((m, 5 + batches * n + 2)), F32)
    out = torch.full((m, batches * n + 3), 9.0, dtype=dtype, device="cuda")
    ops.gemm_batched(out, dev(x, dtype), dev(wt, dtype), batches, m, n, k, batches * k, k, k, n * k, batches * n + 3, n, gate=dev(gate, F32), gate_at=5, gate_batch=n)
    got = out.float().cpu().numpy()
    want = np.einsum("mbk,bnk->mbn", x, wt).reshape(m, batches * n) * plain.sigmoid(gate[:, 5 : 5 + batches * n])
    assert_close(got[:, : batches * n], want, 3e-6 if dtype == F32 else 1e-2, "gated product")
    assert (got[:, batches * n :] == 9.0).all()


# ---- windowed attention with one added to the denominator -----------------------------------------------------------
def attention_mixer(H, G, d, dv, window, dims=None, base=500.0, scaling=(3.0, 1.0, 4.0, 90.0), scale=None):
    rot = {"base": base, "dims": d if dims is None else dims}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": scale or 1.5 / np.sqrt(d), "rot": rot, **({"mask": {"size": window}} if window else {})}


def attention_part(w, m, width, dtype, eps=1e-5, prefix="a."):
    from alofa_b200.config.spec import PartSpec
    from alofa_b200.parts.base import Runtime, build_part

    scaling = {"kind": "wavelength", **m["rot"]["scaling"]} if m["rot"].get("scaling") else None
    rotary = PartSpec("rotary_interleaved", {"dims": m["rot"]["dims"], "base": m["rot"]["base"], "layout": "halves", "scaling": scaling})
    part = build_part("mixer", PartSpec("normed_attention", {"hidden_size": width, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"], "scale": m["scale"],
                                                              "qk_norm": True, "norm_weight": True, "norm_over": "projection", "eps": eps, "position": rotary,
                                                              "window": m["mask"]["size"] if "mask" in m else None, "sink": 0.0}, prefix=prefix), Runtime(torch.device("cuda"), dtype))
    return loaded(part, {k: v for k, v in w.items()}, prefix, dtype, m["heads"] * m["vdim"])


def attention_weights(rng, m, dtype, ones=False, prefix="a."):
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    nq, nk, nv = H * d, G * d, G * dv
    eye = np.eye(nq + nk + nv)
    w = {"q": eye[:nq], "k": eye[nq : nq + nk], "v": eye[nq + nk :], "o": np.eye(H * dv),
         "q.norm": np.ones(nq) if ones else rounded(1 + 0.3 * rng.standard_normal(nq), dtype), "k.norm": np.ones(nk) if ones else rounded(1 + 0.3 * rng.standard_normal(nk), dtype)}
    return {prefix + n: v for n, v in w.items()}, eye.shape[0]


ATTENTIONS = [(F32, 4, 2, 16, 24, 9, 16, 16), (F32, 3, 3, 12, 8, 21, 6, 16), (F32, 2, 1, 10, 30, None, 2, 16), (F32, 1, 1, 8, 130, 2, 8, 16), (F32, 6, 2, 40, 72, 32, 24, 64),
              (BF16, 3, 1, 12, 20, 17, 12, 16), (BF16, 4, 2, 64, 64, 64, 64, 64), (BF16, 4, 1, 64, 64, 1, 32, 64), (BF16, 2, 2, 64, 64, 130, 20, 16), (BF16, 6, 2, 64, 128, 100, 64, 64),
              (BF16, 2, 1, 128, 64, 90, 96, 32), (BF16, 4, 4, 128, 128, 200, 64, 64), (BF16, 20, 1, 32, 48, 40, 32, 16), (BF16, 3, 3, 96, 96, 81, 32, 64), (BF16, 34, 2, 48, 48, None, 24, 48),
              (BF16, 5, 5, 80, 80, 33, 40, 64)]


@pytest.mark.parametrize("dtype,H,G,d,dv,window,dims,page", ATTENTIONS)
def test_windowed_attention_in_prompts_portions_and_decoding(dtype, H, G, d, dv, window, dims, page):
    rng = np.random.default_rng(13)
    m = attention_mixer(H, G, d, dv, window, dims)
    w, width = attention_weights(rng, m, dtype)
    c = window or 50
    lengths = sorted({n for n in [1, 2, page - 1, page, page + 1, c - 1, c, c + 1, c + page, 2 * c + 1, 150 if dtype == F32 else 330] if n > 0})
    rows = [rounded(rng.standard_normal((n, width)), dtype) for n in lengths]
    want = [plain.attention(w, "a.", m, x, 1e-5) for x in rows]
    part = attention_part(w, m, width, dtype)
    for cuts in ((1,), (5, 2, 64, 3, 2, 130)):
        case = Paged(rng, lengths, page, (G, d), (G, dv), dtype, window)
        for what, got in zip(("whole", f"portions of {cuts}"), in_steps(part, case, rows, dtype, cuts)):
            for r, n in enumerate(lengths):
                assert_close(got[r], want[r], KERNEL_TOL[dtype], f"{what}: request of {n} tokens")


PATHS = [(F32, 16, 16), (BF16, 12, 24), (BF16, 64, 64), (BF16, 32, 48), (BF16, 96, 96)]


@pytest.mark.parametrize("dtype,d,dv", PATHS)
@pytest.mark.parametrize("window", [1, 3, 16, 40, 64, 65, 100])
def test_a_key_just_inside_and_just_outside_the_window(dtype, d, dv, window):
    """The last key a far query may not see and the first it may both point the query's way (turned to its place) and hold
    large values: the sum of the right one and no other, in prompts and in decoding."""
    rng = np.random.default_rng(4)
    H, G = 2, 1
    m = attention_mixer(H, G, d, dv, window, scale=1.0, base=20.0)
    w, width = attention_weights(rng, m, dtype, ones=True)
    n = window + 80
    x = rounded(0.2 * rng.standard_normal((n, width)), dtype)
    i = n - 3  # the query
    way = np.sign(rng.standard_normal(d))
    x[i, : H * d] = np.tile(way, H)
    for j, value in ((i - window, 30.0), (i - window + 1, -20.0)):
        back = {k: v for k, v in m["rot"].items()}
        turned = plain.rotate(np.tile(way, (n, 1, 1)), back)  # row t: the way turned by t
        # a key that, turned by j, stands where the query turned by i stands: the way turned by i - j
        x[j, H * d : H * d + d] = turned[i - j, 0]
        x[j, H * d + G * d :] = value
    if window > 1:
        x[i, H * d : H * d + d] = -way  # the query's own key points away
    x = rounded(x, dtype)
    want = plain.attention(w, "a.", m, x, 1e-6)
    wrong = [plain.attention(w, "a.", dict(m, mask={"size": window + a}), x, 1e-6)[i] for a in (1, -1) if window + a > 0]
    assert all(np.abs(want[i] - other).max() > 3.0 for other in wrong), "the test's keys do not stand out"
    part = attention_part(w, m, width, dtype, 1e-6)
    for cuts in ((1,), (7, 2, 64)):
        case = Paged(rng, [n], 64 if d in (64, 96) else 16, (G, d), (G, dv), dtype, window)
        for got in in_steps(part, case, [x], dtype, cuts):
            assert_close(got[0], want, KERNEL_TOL[dtype], f"window {window}, cuts {cuts}")


@pytest.mark.parametrize("dtype,d,dv", PATHS)
@pytest.mark.parametrize("level", [-6.0, 0.0, 4.0])
def test_the_one_in_the_denominator_takes_its_share_once(dtype, d, dv, level):
    """All scores equal ``level``: the output is the values' mean times n e^level / (1 + n e^level), whatever the key blocks
    and splits a row was merged from."""
    rng = np.random.default_rng(7)
    m = attention_mixer(2, 1, d, dv, 300, dims=0, scaling=None, scale=max(abs(level), 1.0) / d)
    w, width = attention_weights(rng, m, dtype, ones=True)
    x = rounded(rng.standard_normal((420, width)), dtype)
    x[:, : 2 * d] = 1.0
    x[:, 2 * d : 3 * d] = np.sign(level) if level else np.where(np.arange(d) % 2, 1.0, -1.0)
    x[:, 3 * d :] += 3.0
    x = rounded(x, dtype)
    want = plain.attention(w, "a.", m, x, 1e-6)
    n = np.minimum(np.arange(420) + 1, 300)
    mean = np.stack([x[max(0, t - 299) : t + 1, 3 * d :].mean(axis=0) for t in range(420)])
    np.testing.assert_allclose(want[:, :dv], mean * (n * np.exp(level) / (1 + n * np.exp(level)))[:, None], rtol=1e-3)
    part = attention_part(w, m, width, dtype, 1e-6)
    for cuts in ((1,), (130, 2)):
        case = Paged(rng, [420], 16, (1, d), (1, dv), dtype, 300)
        for got in in_steps(part, case, [x], dtype, cuts):
            assert_close(got[0], want, KERNEL_TOL[dtype], f"level {level}, cuts {cuts}")


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("halves", [True, False])
@pytest.mark.parametrize("H,G,d,dv,dims,n", [(4, 2, 24, 40, 16, 37), (3, 1, 7, 5, 6, 9), (16, 4, 128, 128, 64, 3), (5, 5, 10, 30, 10, 200), (6, 2, 6, 8, 4, 150), (2, 2, 12, 4, 0, 5)])
def test_norms_over_the_whole_projection_then_a_rotation(dtype, halves, H, G, d, dv, dims, n):
    """q, keys and values from finished sums and from planes of split sums with a bias on top, at positions up to 100,000."""
    from alofa_b200.csrc import ops

    rng = np.random.default_rng(15)
    nq, nk, nv = H * d, G * d, G * dv
    ld = nq + nk + nv
    planes, bias = rounded(rng.standard_normal((3, n, ld)), F32), rounded(rng.standard_normal(ld), F32)
    whole = rounded(planes.sum(axis=0) + bias, F32)
    wq, wk = rounded(1 + 0.2 * rng.standard_normal(nq), F32), rounded(1 + 0.2 * rng.standard_normal(nk), F32)
    slots = rng.permutation(4 * n)[:n].astype(np.int32)
    positions = rng.integers(0, 100_000, n).astype(np.int32)
    freq = rounded(plain.frequencies({"base": 5e4, "dims": max(dims, 2)}), F32)
    # the angle is a product in fp32 (an error of up to one part in 2^24 of 100,000 radians would show otherwise)
    angle = (positions[:, None].astype(np.float32) * freq.astype(np.float32)).astype(np.float64)[:, None, : dims // 2]

    def turned(x, heads):
        x = x.reshape(n, heads, d).copy()
        u, v = (slice(0, dims // 2), slice(dims // 2, dims)) if halves else (slice(0, dims, 2), slice(1, dims, 2))
        a, b = x[..., u].copy(), x[..., v].copy()
        x[..., u], x[..., v] = a * np.cos(angle) - b * np.sin(angle), b * np.cos(angle) + a * np.sin(angle)
        return x.reshape(n, heads * d)

    for sums in (dev(whole, F32), Owed(dev(planes, F32), dev(bias, F32))):
        q = torch.zeros((n, nq), dtype=dtype, device="cuda")
        k, v = torch.zeros((4 * n, G, d), dtype=dtype, device="cuda"), torch.zeros((4 * n, G, dv), dtype=dtype, device="cuda")
        ops.qkv_prepare_rows(q, k, v, sums, dev(slots), dev(wq, F32), dev(wk, F32), 1e-5, positions=dev(positions), freq=dev(freq, F32), rot_dims=dims, halves=halves)
        tol = 4e-6 if dtype == F32 else 1e-2
        assert_close(q.float().cpu(), turned(plain.rms_norm(whole[:, :nq], wq, 1e-5), H), tol, "q")
        assert_close(k.float().cpu().numpy()[slots].reshape(n, nk), turned(plain.rms_norm(whole[:, nq : nq + nk], wk, 1e-5), G), tol, "keys")
        assert_close(v.float().cpu().numpy()[slots].reshape(n, nv), whole[:, nq + nk :], tol, "values")
        unused = np.setdiff1d(np.arange(4 * n), slots)
        assert float(k[unused].abs().max()) == 0.0 and float(v[unused].abs().max()) == 0.0


# ---------------------------------------------------------------------------------------------------
# experts, norms
# ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("E,top,hidden,ff,shared", [(8, 3, 64, 48, 80), (6, 2, 100, 28, None), (5, 1, 128, 64, 32), (4, 4, 64, 16, 12), (32, 8, 256, 40, 96)])
def test_experts_weighted_over_the_chosen_with_a_shared_one(dtype, E, top, hidden, ff, shared):
    from alofa_b200.config.spec import PartSpec
    from alofa_b200.parts.base import Runtime
    from alofa_b200.parts.routed import RoutedExperts

    rng = np.random.default_rng(17)
    w = {"m.router": rounded(3 * rng.standard_normal((E, hidden)) / np.sqrt(hidden), BF16)}
    for name, size in [(f"e{e}.", ff) for e in range(E)] + ([("shared.", shared)] if shared else []):
        w.update({f"m.{name}up": rounded(rng.standard_normal((size, hidden)) / np.sqrt(hidden), BF16), f"m.{name}down": rounded(rng.standard_normal((hidden, size)) / np.sqrt(size), BF16)})
    mlp = {"expert": {"ff": ff}, "router": {"experts": E, "top": top}, **({"shared": {"ff": shared}} if shared else {})}
    part = RoutedExperts(PartSpec("routed_experts", {"hidden_size": hidden, "experts": E, "top": top, "expert_ff": ff, "shared_ff": shared or 0, "activation": "relu_squared",
                                                     "score": "softmax", "renormalize": True}, prefix="m."), Runtime(torch.device("cuda"), dtype))
    part.load({k: dev(v, dtype) for k, v in w.items()})
    for tokens in (1, 7, 64, 150):
        x = rounded(rng.standard_normal((tokens, hidden)), BF16)
        sure = plain.route(w, "m.", mlp["router"], x)[2] > 1e-3
        h = torch.full((tokens, hidden), 5.0, dtype=F32, device="cuda")
        part.forward(Step, dev(x, dtype), h, store=True)
        assert_close(h.cpu().numpy()[sure], plain.routed(w, "m.", mlp, x)[sure], 1e-5 if dtype == F32 else 1.5e-2, f"{tokens} tokens")


@pytest.mark.parametrize("experts,top", [(6, 2), (12, 4), (4, 4), (64, 6), (5, 1)])
def test_router_weights_are_the_softmax_over_the_chosen_logits(experts, top):
    """Also with logits so large that the others' share of a softmax over all experts would not be representable."""
    from alofa_b200.csrc import ops

    rng = np.random.default_rng(11)
    n, hidden = 97, 48
    for gain in (2.0, 60.0):
        x = rounded(rng.standard_normal((n, hidden)), F32)
        w = {"m.router": rounded(gain * rng.standard_normal((experts, hidden)) / np.sqrt(hidden), F32)}
        chosen, weight, margin = plain.route(w, "m.", {"experts": experts, "top": top}, x)
        choice, wgt = torch.empty((n, top), dtype=torch.int32, device="cuda"), torch.empty((n, top), dtype=F32, device="cuda")
        ops.moe_router(choice, wgt, None, dev(x, F32), dev(w["m.router"], F32), experts, top, True, True)
        sure = margin > 1e-4
        assert sure.mean() > 0.9
        got, at = choice.cpu().numpy()[sure], wgt.cpu().numpy()[sure]
        for t, (ids, weights) in enumerate(zip(got, at)):
            want = dict(zip(chosen[sure][t], weight[sure][t]))
            kept = {int(e): float(v) for e, v in zip(ids, weights)}
            assert len(kept) == top and all(abs(kept.get(e, 0.0) - v) <= 2e-5 for e, v in want.items() if v > 1e-30), f"token {t}: {kept} {want}"


@pytest.mark.parametrize("tokens,experts,top,hidden", [(1, 64, 6, 2048), (9, 17, 3, 264), (70, 200, 8, 72), (1100, 33, 2, 136), (5, 4, 2, 100), (3, 20, 2, 8192)])
@pytest.mark.parametrize("x_type,w_type", [(F32, F32), (BF16, F32), (BF16, BF16)])
def test_router_for_few_and_many_tokens_and_experts(tokens, experts, top, hidden, x_type, w_type):
    """Experts dealt over a cluster of blocks and on one block, depths that are and are not multiples of 8, weights in either
    type: 32-bit sums, and a token's logits do not depend on which others come with it."""
    from alofa_b200.csrc import ops

    rng = np.random.default_rng(18)
    x, wr = rounded(rng.standard_normal((tokens, hidden)), x_type), rounded(2 * rng.standard_normal((experts, hidden)) / np.sqrt(hidden), w_type)
    chosen, weight, margin = plain.route({"m.router": wr}, "m.", {"experts": experts, "top": top}, x)

    def run(rows):
        choice, wgt = torch.empty((len(rows), top), dtype=torch.int32, device="cuda"), torch.empty((len(rows), top), dtype=F32, device="cuda")
        ops.moe_router(choice, wgt, None, dev(rows, x_type), dev(wr, w_type), experts, top, True, True)
        return choice.cpu().numpy(), wgt.cpu().numpy()

    choice, wgt = run(x)
    sure = margin > 1e-4
    assert sure.mean() > 0.8 or tokens < 10
    assert (choice[sure] == chosen[sure]).all()
    assert_close(wgt[sure], weight[sure], 1e-5, "weights")
    alone = run(x[tokens // 2 : tokens // 2 + 1])
    assert (alone[0][0] == choice[tokens // 2]).all() and (alone[1][0] == wgt[tokens // 2]).all()


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("tokens,top,experts,tile,hidden,identity", [(1, 1, 4, 64, 24, 0), (8, 6, 64, 128, 256, 0), (37, 3, 5, 64, 30, 2), (128, 8, 40, 128, 8, 0), (129, 8, 70, 128, 20, 3), (3000, 4, 90, 128, 16, 0)])
def test_pairs_are_placed_by_expert_in_one_kernel_or_two(dtype, tokens, top, experts, tile, hidden, identity):
    """Few pairs in one launch, more in two: the same places, tiles and rows (experts past the last are the identity: no row)."""
    from alofa_b200.csrc import ops

    rng = np.random.default_rng(19)
    choice = np.stack([rng.permutation(experts + identity)[:top] if top <= experts else rng.integers(0, experts, top) for _ in range(tokens)]).astype(np.int32)
    tiles = -(-tokens * top // tile) + experts
    x, weight = rounded(rng.standard_normal((tokens, hidden)), dtype), rounded(rng.standard_normal((tokens, top)), F32)
    for scaled in (False, True):
        results = []
        for one in (True, False):
            dest, te = torch.full((tokens, top), -7, dtype=torch.int32, device="cuda"), torch.full((tiles,), -7, dtype=torch.int32, device="cuda")
            xs = torch.zeros((tiles * tile, hidden), dtype=dtype, device="cuda")
            w = dev(weight, F32) if scaled else None
            if one:
                assert ops.moe_place(xs, dest, te, dev(choice), dev(x, dtype), w, experts, tile, top) == (tokens * top <= 1024)
            if not one or tokens * top > 1024:
                ops.moe_sort(dest, te, dev(choice), experts, tile)
                ops.moe_scatter(xs, dev(x, dtype), w, dest, top)
            results.append((dest.cpu().numpy().ravel(), te.cpu().numpy(), xs.float().cpu().numpy()))
        d, te, xs = results[0]
        assert all((a == b).all() for a, b in zip(results[0], results[1]))
        flat, rows = choice.ravel(), np.repeat(x, top, axis=0) * (weight.reshape(-1, 1) if scaled else 1.0)
        real = flat < experts
        assert (d[~real] == -1).all() and len(set(d[real].tolist())) == real.sum() and (te[d[real] // tile] == flat[real]).all()
        for e in range(experts):
            assert (np.diff(d[flat == e]) == 1).all()
        used = te[te >= 0]
        assert (np.diff(used) >= 0).all() and (te[len(used):] == -1).all()
        assert_close(xs[d[real]], rows[real], 1e-6 if dtype == F32 else 8e-3, "rows")


@pytest.mark.parametrize("tokens,top,hidden", [(1, 1, 30), (5, 6, 2048), (70, 32, 100), (9, 2, 516)])
def test_combine_adds_choices_in_order_and_the_shared_output(tokens, top, hidden):
    from alofa_b200.csrc import ops

    rng = np.random.default_rng(20)
    ys, shared, y0 = (rounded(rng.standard_normal(s), F32) for s in ((tokens * top + 3, hidden), (tokens, hidden), (tokens, hidden)))
    dest, weight = rng.permutation(tokens * top + 3)[: tokens * top].reshape(tokens, top).astype(np.int32), rounded(rng.standard_normal((tokens, top)), F32)
    for w, sh, add in ((weight, shared, False), (None, None, True), (weight, None, True)):
        y = dev(y0, F32)
        ops.moe_combine(y, dev(ys, F32), dev(dest), dev(w, F32) if w is not None else None, dev(sh, F32) if sh is not None else None, None, top, add=add)
        want = (ys[dest] * (w[:, :, None] if w is not None else 1.0)).sum(axis=1) + (sh if sh is not None else 0.0) + (y0 if add else 0.0)
        assert_close(y.cpu(), want, 3e-6, "combined")


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("rows,width", [(1, 96), (9, 100), (7, 30), (300, 1024)])
def test_norm_with_its_weight_stored_less_one(dtype, rows, width):
    """Stored numbers so small that one more than them, rounded to bfloat16, would be one."""
    from alofa_b200.config.spec import PartSpec
    from alofa_b200.parts.base import Runtime, build_part

    class Ctx(Step):
        def __init__(self):
            pass

        stream_of = staticmethod(lambda h: None)
        take_pending = staticmethod(lambda h: None)

    rng = np.random.default_rng(12)
    stored = rounded(0.003 * rng.standard_normal(width), BF16)
    part = build_part("norm", PartSpec("rmsnorm", {"size": width, "eps": 1e-5, "weight_name": "n", "weight_offset": 1.0}), Runtime(torch.device("cuda"), dtype))
    part.load({"n": dev(stored, BF16)})
    assert_close(part.weight.cpu(), 1.0 + stored, 1e-7, "weight")
    x = rounded(rng.standard_normal((rows, width)), F32)
    assert_close(part.forward(Ctx(), dev(x, F32)).float().cpu(), plain.offset_norm(x, stored, 1e-5), 2e-6 if dtype == F32 else 8e-3, "rows")


# ---------------------------------------------------------------------------------------------------
# whole models
# ---------------------------------------------------------------------------------------------------
LENGTHS = {"A": [1, 2, 18, 19, 64, 65, 129, 200], "B": [3, 16, 17, 33, 80, 131], "C": [5, 63, 190, 257], "D": [2, 37, 150, 300], "E": [4, 69, 70, 189, 330]}
DECODED = 12


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    base = tmp_path_factory.mktemp("nugopel_gpu")
    return {name: tiny.write(base / name, name, seed=10 + i) for i, name in enumerate(tiny.CONFIGS)}


def make_requests(name):
    reqs, prompts = {}, {}
    for i, n in enumerate(LENGTHS[name]):
        reqs[f"r{i}"] = tiny.tokens(name, n + DECODED, seed=i)
        prompts[f"r{i}"] = n
    return reqs, prompts


@pytest.fixture(scope="module")
def plain_logits(folders):
    out = {}
    for name, folder in folders.items():
        w, cfg = plain.load(folder)
        logits, sure = {}, {}
        for rid, toks in make_requests(name)[0].items():
            logits[rid], margins = plain.forward(w, cfg, toks, margins=True)
            sure[rid] = plain.sure_prefix(margins, 0.15)
        out[name] = (logits, sure)
    return out


def runner_for(folder, dtype, block, pages, max_requests=4, graphs=True):
    from alofa_b200.engine.loading import load_model
    from alofa_b200.engine.step import StepRunner

    model, *_ = load_model(folder, dtype)
    return StepRunner(model, block_size=block, num_pages=pages, max_requests=max_requests, max_tokens=pages * block, max_step_tokens=512, cuda_graphs=graphs)


def assert_most_close(errors, tol, what):
    errors = np.asarray(errors)
    assert (errors > tol).mean() <= 0.25 and np.median(errors) <= tol / 3, \
        f"{what}: {(errors > tol).sum()} of {len(errors)} positions beyond {tol:.1e}, median {np.median(errors):.3e}, worst {errors.max():.3e}"


def compare(steps, outputs, want, vocab, tol, what, sure=None):
    """Every position within ``tol`` in 32-bit.  In bfloat16 strictly up to a request's first close call of a router
    (``sure``: two scores within rounding of one another, where bfloat16 may rightly take the other expert); over all
    positions three quarters keep the bound and the median a third of it: a lost state, a wrong key or page moves
    every position by order one."""
    got = replay.collect(steps, outputs, vocab)
    errors = []
    for rid, rows in got.items():
        ref = want[rid][: len(rows)]
        assert rows.shape == ref.shape, f"{what} {rid}: {rows.shape} vs {ref.shape}"
        err = np.abs(rows - ref).max(axis=-1) / max(1.0, float(np.abs(ref).max()))
        n = len(rows) if sure is None else min(len(rows), sure[rid])
        if n:
            assert err[:n].max() <= tol, f"{what} {rid}: position {int(err[:n].argmax())} differs by {err[:n].max():.3e} > {tol:.1e}"
        errors.append(err)
    assert_most_close(np.concatenate(errors), tol, what)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_whole_decoded_portions_and_mixed_batches(folders, plain_logits, name, dtype):
    """The same requests whole, with the last tokens decoded one by one, in portions down to two tokens, and mixed
    (portions beside single tokens, four live at most, four state slots) in a pool that holds two of the longest: pages
    and slots are given back and used again.  Every position against plain."""
    reqs, prompts = make_requests(name)
    vocab = tiny.CONFIGS[name]["vocab"]
    block = 16 if name in ("B", "D") else 64
    per_request = -(-max(len(t) for t in reqs.values()) // block)
    schedules = {
        "whole": (replay.whole(reqs), per_request),
        "decoded": (replay.tail_decoded(reqs, tail=DECODED + 20), per_request),
        "portions": (replay.portions(reqs), per_request),
        "mixed": (replay.mixed(reqs, prompts, 2 * per_request * block + block, block, seed=3), 2 * per_request + 1),
    }
    for what, (steps, pages) in schedules.items():
        runner = runner_for(folders[name], dtype, block, pages, max_requests=4)
        out = replay.run_inprocess(runner, steps)
        compare(steps, out, plain_logits[name][0], vocab, TOL[dtype], f"{name}/{dtype}/{what}", sure=plain_logits[name][1] if dtype == "bfloat16" else None)
        assert set(runner.manager.free_pages()) == {pages} and runner.manager.live_requests() == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C", "D", "E"])
def test_long_decoding_from_the_first_token(folders, name, dtype):
    """One prompt token, then 170 tokens one by one (past page borders, past every window's edge and the kept tokens), two
    requests side by side that started 40 steps apart; decode steps are replayed as graphs."""
    from alofa_b200.engine.step import StepEntry

    w, cfg = plain.load(folders[name])
    a, b = tiny.tokens(name, 171, seed=50), tiny.tokens(name, 131, seed=51)
    (want_a, ma), (want_b, mb) = plain.forward(w, cfg, a, margins=True), plain.forward(w, cfg, b, margins=True)
    sure_a, sure_b = (plain.sure_prefix(ma, 0.15), plain.sure_prefix(mb, 0.15)) if dtype == "bfloat16" else (171, 131)
    runner = runner_for(folders[name], dtype, 16, 22, max_requests=2)
    sa, sb, errors = runner.admit(0), None, []
    for i in range(171):
        entries = [StepEntry(sa, [a[i]], [0])]
        if i >= 40:
            if sb is None:
                sb = runner.admit(1)
            entries.append(StepEntry(sb, [b[i - 40]], [0]))
        rows = runner.forward(entries).float().cpu().numpy()
        for row, want, k, sure, who in ((rows[0], want_a, i, sure_a, "first"),) + (((rows[1], want_b, i - 40, sure_b, "second"),) if i >= 40 else ()):
            if k < sure:
                assert_close(row, want[k], TOL[dtype], f"{who} request, token {k}")
            errors.append(np.abs(row - want[k]).max() / max(1.0, float(np.abs(want).max())))
    assert_most_close(errors, TOL[dtype], "long decoding")
    runner.check_status()
    assert runner.manager.defects() == 0


def test_batches_and_cuts_do_not_change_a_request(folders):
    """float32: a request's logits in portions and in a mixed batch equal, to rounding of the sums' order, those it gets alone and whole."""
    name = "D"
    reqs, prompts = make_requests(name)
    vocab = tiny.CONFIGS[name]["vocab"]
    alone = replay.collect(replay.whole(reqs), replay.run_inprocess(runner_for(folders[name], "float32", 16, 20), replay.whole(reqs)), vocab)
    for what, steps, pages in (("portions", replay.portions(reqs), 20), ("mixed", replay.mixed(reqs, prompts, 700, 16, seed=9), 44)):
        other = replay.collect(steps, replay.run_inprocess(runner_for(folders[name], "float32", 16, pages, max_requests=4), steps), vocab)
        for rid in reqs:
            assert np.abs(alone[rid] - other[rid]).max() <= 1e-5 * max(1.0, np.abs(alone[rid]).max()), f"{what} {rid}"


def test_pages_behind_the_window_are_given_back_and_the_latents_stay(folders):
    """After a long prompt a request of configuration D holds the windows' pages in the windowed groups and every page of the
    latent that two layers read, of which there is one cache."""
    from alofa_b200.engine.step import StepEntry

    runner = runner_for(folders["D"], "bfloat16", 16, 25)
    slot = runner.admit(0)
    runner.forward([StepEntry(slot, tiny.tokens("D", 390, seed=3), [389])])
    runner.check_status()
    assert sorted(g.window or 0 for g in runner.group_specs) == [0, 37, 100]
    for gi, g in enumerate(runner.group_specs):
        table = runner.manager.block_table(slot, gi)
        passed = (390 - g.window + 1) // 16 if g.window else 0
        assert (table[:passed] < 0).all() and (table[passed : -(-390 // 16)] >= 0).all()
    assert len(runner.model.cache_plan()) == 3


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_the_stream_after_every_layer(folders, name):
    """float32: the residual stream after each layer."""
    import alofa_b200.parts.block as block
    from alofa_b200.engine.step import StepEntry

    w, cfg = plain.load(folders[name])
    ids = tiny.tokens(name, 30, seed=77)
    _, want = plain.forward(w, cfg, ids, streams=True)
    seen, original = [], block.SandwichResidual.forward

    def recording(self, ctx, h, cache, writes=True):
        original(self, ctx, h, cache, writes)
        ctx.flush_pending()
        seen.append(h.double().cpu().numpy())

    block.SandwichResidual.forward = recording
    try:
        runner = runner_for(folders[name], "float32", 64, 1, graphs=False)
        runner.forward([StepEntry(runner.admit(0), ids, [0])])
    finally:
        block.SandwichResidual.forward = original
    assert len(seen) == len(want) == len(cfg["layers"])
    for k, (got, ref) in enumerate(zip(seen, want)):
        assert_close(got, ref, TOL["float32"], f"after layer {k}")


@pytest.mark.parametrize("name", list(tiny.CONFIGS))
def test_greedy_generation_through_the_engine(folders, name):
    """Engine.generate (scheduler, chunked prefill, decode graphs): float32 tokens equal plain greedy; bfloat16 tokens
    are each within rounding of the plain maximum, up to the first close call of a router."""
    from alofa_b200.engine.engine import Engine

    w, cfg = plain.load(folders[name])
    prompts = [tiny.tokens(name, n, seed=200 + i) for i, n in enumerate([1, 7, 40, 90, 18])]
    want = [plain.greedy(w, cfg, p, 6) for p in prompts]
    eng = Engine(str(folders[name]), dtype="float32", block_size=16, max_batch=3, token_budget=48, max_chunk=32, max_tokens=128)
    assert eng.generate(prompts, max_new_tokens=6) == want
    assert eng.stats()["defects"] == 0
    eng16 = Engine(str(folders[name]), dtype="bfloat16", block_size=16, max_batch=3, token_budget=48, max_chunk=32, max_tokens=128)
    for p, out in zip(prompts, eng16.generate(prompts, max_new_tokens=6)):
        seq = list(p)
        for tok in out:
            logits, margins = plain.forward(w, cfg, seq, margins=True)
            if plain.sure_prefix(margins, 0.15) < len(seq):
                break
            row = logits[-1]
            assert row.max() - row[tok] <= 8e-2 * max(1.0, float(np.abs(row).max())), "a bfloat16 token is not near the plain maximum"
            seq.append(tok)
    eng16.runner.check_status()


def test_the_programs_take_the_architecture(folders, tmp_path):
    """bin/trace_run replays a schedule and bin/generate generates, both choosing the model by config.json."""
    name = "C"
    reqs, _ = make_requests(name)
    reqs = {k: reqs[k] for k in ("r0", "r2")}
    w, cfg = plain.load(folders[name])
    want = {rid: plain.forward(w, cfg, t) for rid, t in reqs.items()}
    steps = replay.portions(reqs, sizes=(40, 2, 3, 64, 1))
    out = replay.run_trace_program(folders[name], "float32", steps, tmp_path / "out", 512)
    compare(steps, out, want, cfg["vocab"], TOL["float32"], "trace_run")
    prompt = tiny.tokens(name, 12, seed=5)
    done = subprocess.run([sys.executable, str(replay.ROOT / "bin" / "generate"), "--model", str(folders[name]), "--dtype", "float32", "--prompt-ids",
                           ",".join(map(str, prompt)), "--max-new-tokens", "5", "--max-tokens", "64", "--json"], capture_output=True, text=True, timeout=600)
    assert done.returncode == 0, done.stderr[-2000:]
    assert json.loads(done.stdout.strip().splitlines()[-1])["out_ids"] == [plain.greedy(w, cfg, prompt, 5)]
