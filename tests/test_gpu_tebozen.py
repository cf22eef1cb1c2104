"""The Tebozen design in the engine against the plain implementation (``plain_tebozen``): every mechanism alone, whole
prompts against token-by-token decoding, portions down to two tokens, batches of unequal requests, slots and pages that are
used again, keys far away, at page borders and just inside and outside every window, the first tokens, memories that last and
that fade, long decoding, sizes that are 1 or equal, generation through the library's own loop, and trace replay (needs a
B200)."""
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_tebozen as pz
import tebozen_helpers as th
from helpers import FP32_TOL, run_trace
from questwend_b200.cache import CacheManager
from questwend_b200.engine.engine import Engine, StepEntry, build_step_context
from questwend_b200.kernels import ops
from questwend_b200.parts import PartSpec, Runtime, build_part

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda:0")
DTYPES = [torch.float32, torch.bfloat16]
BF16_RMS_TOL = 0.03         # bfloat16 engine against the plain implementation that rounds the products' operands and what the
                            # cache holds: root mean square of the difference over the reference's
EPS = 1e-5
WIDTH = 48


def close(got, ref, dtype, tol=FP32_TOL):
    got, ref = np.asarray(got, dtype=np.float64), np.asarray(ref, dtype=np.float64)
    if dtype == torch.float32:
        return np.abs(got - ref).max() <= tol * np.abs(ref).max()
    return np.sqrt(np.mean((got - ref) ** 2)) <= BF16_RMS_TOL * np.sqrt(np.mean(ref ** 2))


def rows_close(got, ref, dtype):
    """The same for a whole model's logits.  In bfloat16 a router's choice between two experts with nearly equal scores can
    fall either way, and a difference of two maps that nearly cancel is normed: a row in twenty may be off, every other one is
    held to a wider tolerance by itself, and the row in the middle to the tolerance."""
    if dtype == torch.float32:
        return close(got, ref, dtype)
    err = np.sqrt(np.mean((np.asarray(got) - ref) ** 2, axis=-1)) / np.sqrt(np.mean(ref ** 2))
    return np.sum(err > 4 * BF16_RMS_TOL) <= len(err) // 20 and np.median(err) <= BF16_RMS_TOL


def dev(a, dtype=torch.float32):
    return torch.from_numpy(np.ascontiguousarray(a)).to(dtype).to(DEV)


def f32(a):
    return np.float32(a).astype(np.float64)


def host(t):
    return t.double().cpu().numpy()


# ----------------------------------------------------------------------------- the matrix memory's kernels
class Steps:
    """What the recurrence reads of a step: B sequences with these numbers of tokens, in these slots."""

    def __init__(self, counts, slots):
        self.cu_seqlens, self.slots = dev(np.concatenate([[0], np.cumsum(counts)]), torch.int32), dev(slots, torch.int32)
        self.n_seqs, self.max_new, self.single_token = len(counts), max(counts), all(c == 1 for c in counts)


def draw_memory(rng, n, H, K, P, kind):
    """q, k, v and raw gates of one sequence; ``kind``: what the gates do."""
    q, k, v = (f32(rng.standard_normal((n, H, d))) for d in (K, K, P))
    i, f = {"mixed": (rng.normal(0, 2, (n, H)), rng.normal(2, 2, (n, H))), "lasting": (rng.normal(-1, 1, (n, H)), rng.uniform(7, 12, (n, H))),
            "fading": (rng.normal(0, 1, (n, H)), rng.uniform(-6, -3, (n, H))),
            "high": (np.where(np.arange(n)[:, None] == 2, 40.0, rng.normal(0, 1, (n, H))), rng.uniform(7, 12, (n, H)))}[kind]
    if kind == "high":          # a write far above all others whose level then stays, at a key that no query reads: the running
        q, k = np.abs(q), np.abs(k)     # maximum keeps it, so that e^-m and the small number beside it make the denominator
        q[:, :, 0], k[:, :, 0] = 0.0, 0.0
        k[2:3], k[2:3, :, 0] = 0.0, 1.0
    return q, k, v, f32(i), f32(f)


def run_memory(seqs, H, K, P, cap, plan, bias, chunked=None, slots=None, write=True, state=None):
    """``plan``: steps, each a list of token counts per sequence (0: not in the step)."""
    i_b, f_b = bias
    n_slots = len(seqs) + 2
    slots = slots or list(range(1, len(seqs) + 1))
    st, m = state or (torch.zeros((n_slots, H, P + 1, K), device=DEV), torch.zeros((n_slots, H, P + 1), device=DEV))
    at, got = [0] * len(seqs), [[] for _ in seqs]
    for counts in plan:
        who = [s for s, c in enumerate(counts) if c]
        rows = []
        for s in who:
            q, k, v, i, f = (a[at[s]:at[s] + counts[s]].reshape(counts[s], -1) for a in seqs[s])
            rows.append(np.concatenate([q, k, v, np.full((counts[s], 3), 7.0), i, f], axis=1))
        proj = dev(np.concatenate(rows))
        n_qkv = H * (2 * K + P)
        raw, div = ops.mlstm_scan(proj, n_qkv + 3, n_qkv + 3 + H, dev(i_b), dev(f_b), cap, st, m, Steps([counts[s] for s in who], [slots[s] for s in who]),
                                  H, K, P, K ** -0.5, pz.TINY, write_state=write, chunked=chunked)
        out = host(raw).reshape(-1, H, P) / host(div)[:, :, None]
        off = 0
        for s in who:
            got[s].append(out[off:off + counts[s]])
            off += counts[s]
            at[s] += counts[s]
    return [np.concatenate(g) for g in got], st, m


def memory_oracle(seq, cap, bias):
    q, k, v, i, f = seq
    one, none = np.eye(i.shape[1]), np.zeros((i.shape[1],) * 2)
    li, lf = pz.gates(np.concatenate([i, f], axis=1), {"gate_cap": cap}, {"i": np.concatenate([one, none], 1), "f": np.concatenate([none, one], 1),
                                                                          "i.b": bias[0], "f.b": bias[1]}, "")
    return np.stack([pz.matrix_memory(q[:, h] / np.sqrt(q.shape[2]), k[:, h], v[:, h], li[:, h], lf[:, h]) for h in range(i.shape[1])], axis=1)


@pytest.mark.parametrize("kind", ["mixed", "lasting", "fading", "high"])
@pytest.mark.parametrize("H, K, P", [(1, 1, 1), (3, 8, 12), (2, 20, 6), (2, 40, 72), (1, 64, 136), (2, 130, 33), (1, 256, 200), (1, 500, 20), (5, 12, 64)])
def test_matrix_memory_in_every_form(H, K, P, kind):
    """The scan, the chunked form and single tokens over sequences of unequal lengths (at, below and above the chunk of 64),
    whole, in portions and mixed, against the recurrence in float64; the state of other slots stays as it was."""
    if kind == "high" and K == 1:
        return                                              # its one key row is the one that no query reads
    rng = np.random.default_rng(H * 1000 + K + P)
    lens, cap = [200, 1, 64, 129], 15.0 if kind == "high" else 6.0
    seqs = [draw_memory(rng, n, H, K, P, kind) for n in lens]
    bias = f32(0.5 * rng.standard_normal(H)), f32(0.5 * rng.standard_normal(H))
    refs = [memory_oracle(s, cap, bias) for s in seqs]
    cuts = [[63, 1, 1, 65], [2, 0, 63, 64], [135, 0, 0, 0]]
    plans = [([lens], False), ([lens], True), (cuts, True), (cuts, False), ([[150, 1, 40, 100]] + [[1, 0, 1, 1]] * 24 + [[26, 0, 0, 5]], None)]
    ends = []
    for plan, chunked in plans:
        got, st, m = run_memory(seqs, H, K, P, cap, plan, bias, chunked)
        for g, r in zip(got, refs):
            assert np.abs(g - r).max() <= 3e-5 * np.abs(r).max(), (plan[0], chunked, np.abs(g - r).max() / np.abs(r).max())
        assert not st[0].any() and not st[-1].any() and not m[0].any() and (m[1:-1].amax(-1) == m[1:-1].amin(-1)).all()
        ends.append((st, m))
    for st, m in ends[1:]:
        assert (m - ends[0][1]).abs().max() <= 1e-5 * (1 + m.abs().max())
        assert (st - ends[0][0]).abs().max() <= 1e-4 * ends[0][0].abs().max()
    if kind == "high":                                      # the oracle moves when the maximum or the small number is left out
        tiny, pz.TINY = pz.TINY, 0.0
        moved = memory_oracle(seqs[0], cap, bias)
        pz.TINY = tiny
        assert np.abs(moved - refs[0]).max() > 0.01 * np.abs(refs[0]).max()
    if kind == "lasting":                                   # the first tokens are still read at the end
        q, k, v, i, f = seqs[0]
        gone = memory_oracle((q, k, np.concatenate([-v[:5], v[5:]]), i, f), cap, bias)
        assert np.abs(gone[-1] - refs[0][-1]).max() > 1e-3 * np.abs(refs[0][-1]).max()


def test_matrix_memory_that_only_reads():
    """``write_state`` False leaves state and maximum as they are, in every form."""
    rng = np.random.default_rng(3)
    seqs, bias = [draw_memory(rng, n, 2, 8, 12, "mixed") for n in (100, 70)], (np.zeros(2), np.zeros(2))
    _, st, m = run_memory(seqs, 2, 8, 12, 6.0, [[99, 69]], bias)
    before = st.clone(), m.clone()
    for counts, chunked in (([100, 70], True), ([100, 70], False), ([1, 1], None)):
        run_memory(seqs, 2, 8, 12, 6.0, [counts], bias, chunked, write=False, state=(st, m))
        assert torch.equal(st, before[0]) and torch.equal(m, before[1])


# ----------------------------------------------------------------------------- score maps with windows and gates
def maps_oracle(q, k, v, before, maps, scale, window, lam, norm_out, eps, out_scale, gate):
    n, H = q.shape[:2]
    G = k.shape[1]
    back = before + np.arange(n)[:, None] - np.arange(len(k))[None, :]
    seen = (back >= 0) & (back < (window or len(k)))
    out = np.zeros((n, H, v.shape[2]))
    for h in range(H):
        a = [pz.softmax(q[:, h, m] @ k[:, h // (H // G), m].T * scale, seen) @ v[:, h // (H // G)] for m in range(maps)]
        o = a[0] - lam * a[1] if maps == 2 else a[0]
        out[:, h] = (pz.unit_rms(o, eps) * out_scale if norm_out else o) * (1.0 if gate is None else pz.sigmoid(gate[:, h:h + 1]))
    return out.reshape(n, -1)


@pytest.mark.parametrize("maps, H, G, dim, vdim, window, gated", [
    (2, 4, 2, 16, 32, 20, True), (2, 2, 1, 64, 128, 64, True), (2, 6, 2, 48, 88, 65, False), (2, 2, 2, 32, 136, 130, True), (2, 3, 1, 16, 40, 1, True),
    (1, 4, 2, 32, 24, 63, True), (1, 4, 2, 64, 64, 70, False), (2, 8, 2, 80, 64, 2, True), (1, 2, 2, 160, 256, 100, True), (2, 2, 1, 128, 128, 0, True)])
def test_windows_and_gates_of_score_maps(maps, H, G, dim, vdim, window, gated):
    """Unequal prompts that go on from cached tokens, and single tokens, over shuffled pages whose other rows hold large
    numbers; for many queries a key that stands out sits just inside or just outside the window, at position 0 or at a page's
    border.  bfloat16 kernels against float64 attention on the same inputs."""
    rng = np.random.default_rng(dim + vdim + window)
    scale, lam, out_scale = dim ** -0.5, 0.35, 0.6
    for before, new in (([0, 37, 200, 64, 5], [150, 91, 130, 1, 64]), ([63, 64, 300, 0, 19], [1, 1, 1, 1, 1])):
        B, total = len(new), [a + b for a, b in zip(before, new)]
        width = max(-(-t // 64) for t in total)
        order = rng.permutation(B * width + 3)
        table = np.zeros((B, width), dtype=np.int32)
        k_pool = torch.full((len(order), G, 64, maps * dim), 30.0, dtype=torch.bfloat16, device=DEV)
        v_pool = torch.full((len(order), G, 64, vdim), -500.0, dtype=torch.bfloat16, device=DEV)
        qs, ks, vs, gs = [], [], [], []
        for b in range(B):
            L = total[b]
            k, v = pz.round_bf16(rng.standard_normal((L, G, maps, dim))), pz.round_bf16(rng.standard_normal((L, G, vdim)))
            q = pz.round_bf16(rng.standard_normal((new[b], H, maps, dim)))
            for i in range(0, new[b], 7):
                pos = before[b] + i
                first = max(0, pos - window + 1) if window else 0
                for j in (first, first - 1, 0, 64 * (pos // 64), 64 * (pos // 64) - 1)[(i + b) % 5:(i + b) % 5 + 1]:
                    if 0 <= j < L:
                        k[j] = pz.round_bf16(3.0 * q[i, ::H // G])
            table[b, :-(-L // 64)] = order[b * width:b * width + -(-L // 64)]
            for page in range(-(-L // 64)):
                rows = slice(64 * page, min(64 * page + 64, L))
                k_pool[table[b, page], :, :rows.stop - rows.start] = dev(k[rows].reshape(-1, G, maps * dim).transpose(1, 0, 2), torch.bfloat16)
                v_pool[table[b, page], :, :rows.stop - rows.start] = dev(v[rows].transpose(1, 0, 2), torch.bfloat16)
            qs.append(q), ks.append(k), vs.append(v), gs.append(f32(2 * rng.standard_normal((new[b], H))))
        cu = np.concatenate([[0], np.cumsum(new)])
        ctx = SimpleNamespace(single_token=max(new) == 1, n_seqs=B, max_new=max(new), max_len=max(total), cu_seqlens=dev(cu, torch.int32),
                              pos0=dev(before, torch.int32), seq_len=dev(total, torch.int32))
        gate = dev(np.concatenate([np.concatenate([np.full((n, 5), 9.0), g, np.full((n, 2), 9.0)], 1) for n, g in zip(new, gs)])) if gated else None
        q_all = dev(np.concatenate(qs).reshape(-1, H, maps * dim), torch.bfloat16)
        want = np.concatenate([maps_oracle(qs[b], ks[b], vs[b], before[b], maps, scale, window, lam, maps == 2, EPS, out_scale, gs[b] if gated else None)
                               for b in range(B)])
        for impl in ("auto", "plain"):
            got = host(ops.maps_attention(q_all, k_pool, v_pool, dev(table, torch.int32), ctx, maps, scale, window=window, lam=lam, norm_out=maps == 2,
                                          eps=EPS, out_scale=out_scale, gate=gate, gate_col0=5, impl=impl))
            ops.gemm_tc_check(DEV)
            rms = np.sqrt(np.mean(want ** 2))
            assert np.sqrt(np.mean((got - want) ** 2)) <= 0.012 * rms, (impl, new)
            assert np.abs(got - want).max() <= 0.08 * np.abs(want).max(), (impl, new)


# ----------------------------------------------------------------------------- the experts and their weights
MOES = [th.moe(), th.moe(ff=24, experts=9, top=4, shared=16), th.moe(ff=16, experts=5, top=1, shared=72), th.moe(ff=10, experts=3, top=3, shared=30),
        th.moe(shared=0), th.moe(ff=8, experts=1, top=1, shared=1), th.moe(ff=264, experts=3, top=1, shared=520), th.moe(ff=7, experts=12, top=5, shared=3)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mlp", MOES)
def test_experts_with_weights_on_their_inputs(mlp, dtype):
    """Few tokens (experts streamed) and many (sorted by expert), written and added onto a sum; widths that are and are not
    multiples of 8."""
    from questwend_b200.config.registry import config_from_dict
    from questwend_b200.models.tebozen import _feed_forward
    r16 = dtype == torch.bfloat16
    for width in (64, 36, 27):
        cfgd = th.config([(th.memory(), mlp)], width=width)
        w = th.draw_weights(cfgd, 5)
        spec = _feed_forward(config_from_dict(cfgd).layers[0]["mlp"], width)
        part = build_part("feed_forward", PartSpec(spec.kind, spec.params, prefix="l0.mlp."), Runtime(DEV, dtype))
        part.bind({t.name: dev(w[t.name], dtype if t.role == "matrix" else torch.float32) for t in part.tensors()})
        rng = np.random.default_rng(6)
        for T in (1, 2, 5, 16, 17, 40, 300):
            x = pz.round_bf16(rng.standard_normal((T, width)))
            ok = pz.route_margin(pz.product(x, w["l0.mlp.router"], r16), mlp["router"]["top"]) > 1e-4
            want = pz.experts(x, mlp, w, "l0.mlp.", r16)
            got = host(part.forward(dev(x, dtype), None))
            assert close(got[ok], want[ok], dtype), (width, T)
            y = f32(rng.standard_normal((T, width)))
            onto = dev(y)
            assert part.forward(dev(x, dtype), None, residual=onto) is None
            assert np.abs(host(onto) - (y + got)).max() <= 1e-5 * np.abs(got).max()


@pytest.mark.parametrize("dtype", DTYPES)
def test_gated_experts_take_weights_on_inputs_too(dtype):
    rng = np.random.default_rng(2)
    E, D, F, top = 5, 32, 24, 2
    up, down = pz.round_bf16(rng.standard_normal((E, 2 * F, D)) / 6), pz.round_bf16(rng.standard_normal((E, D, F)) / 5)
    for T in (3, 50):
        x, weight = pz.round_bf16(rng.standard_normal((T, D))), f32(rng.uniform(0.2, 1.5, (T, top)))
        chosen = np.stack([rng.permutation(E)[:top] for _ in range(T)])
        want = np.zeros((T, D))
        for t in range(T):
            for c, s in zip(chosen[t], weight[t]):
                g, u = np.split(up[c] @ (s * x[t]), 2)
                want[t] += down[c] @ (g * pz.sigmoid(g) * u)
        args = dev(x, dtype), dev(up, dtype), dev(down, dtype), dev(chosen, torch.int32), dev(weight)
        assert close(host(ops.moe_experts(*args, weight_on_input=True)), want, dtype)
        if dtype == torch.bfloat16:
            assert close(host(ops.moe_experts_grouped(*args, weight_on_input=True)), want, dtype)


# ----------------------------------------------------------------------------- the mixers alone
class Mixers:
    """Layers' mixers over one cache: the first one's, and for latent attention also of a layer that reads its rows."""

    def __init__(self, layers, dtype, w, n_tokens, n_seqs, longest, width=WIDTH):
        from questwend_b200.config.registry import config_from_dict
        from questwend_b200.models.tebozen import _mixer
        cfgd = th.config([(l, None) for l in layers], width=width, eps=EPS)
        self.dtype, self.parts, rt = dtype, [], Runtime(DEV, dtype)
        for i, layer in enumerate(config_from_dict(cfgd).layers):
            spec, position = _mixer(layer["type"], layer["mixer"], width, EPS)
            part = build_part("mixer", PartSpec(spec.kind, spec.params, prefix=f"l{i}.mix."), rt,
                              position=build_part("position", position, rt) if position else None)
            part.bind({t.name: dev(w[t.name], dtype if t.role == "matrix" else torch.float32) for t in part.tensors()})
            self.parts.append(part)
        self.cache = CacheManager([(p.kv_spec(), p.state_spec(), l["mixer"].get("kv_from")) for p, l in zip(self.parts, layers)],
                                  n_tokens + 64 * n_seqs, n_seqs + 1, longest + 64, dtype, DEV)
        self.units = [self.cache.unit_cache(i) for i in range(len(layers))]

    def run(self, xs, plan):
        """``plan``: a list of steps, each a list of token counts per sequence (0: the sequence sits the step out).  Returns,
        for every mixer, each sequence's outputs in order."""
        slots = self.cache.open(len(xs))
        at = [0] * len(xs)
        got = [[[] for _ in xs] for _ in self.parts]
        for counts in plan:
            who = [i for i, c in enumerate(counts) if c]
            ctx = build_step_context(self.cache, [StepEntry(slots[i], [0] * counts[i], []) for i in who], 10 ** 6, DEV)[0]
            x = dev(np.concatenate([xs[i][at[i]:at[i] + counts[i]] for i in who]), self.dtype)
            for k, (part, unit) in enumerate(zip(self.parts, self.units)):
                out, off = host(part.forward(x, ctx, unit)), 0
                for i in who:
                    got[k][i].append(out[off:off + counts[i]])
                    off += counts[i]
            for i in who:
                self.cache.advance(slots[i], counts[i])
                at[i] += counts[i]
        assert all(a == len(x) for a, x in zip(at, xs))
        self.cache.close(slots)
        return [[np.concatenate(g) for g in per] for per in got]


def oracle(layers, xs, w, r16):
    out, rows = [], {}
    for i, layer in enumerate(layers):
        px, m = f"l{i}.mix.", layer["mixer"]
        if layer["type"] == "latent_attention":
            both = [pz.latent_attention(x, m, w, px, EPS, r16, rows=rows[m["kv_from"]][n] if "kv_from" in m else None) for n, x in enumerate(xs)]
            out.append([b[0] for b in both])
            rows[i] = [b[1] for b in both]
        else:
            out.append([{"mlstm": pz.mlstm, "attention": pz.attention}[layer["type"]](x, m, w, px, EPS, r16) for x in xs])
    return out


LAYERS = [[th.memory()], [th.memory(heads=2, dim=20, vdim=6, cap=9.0)], [th.memory(heads=1, dim=1, vdim=3, cap=1.0)], [th.memory(heads=2, dim=72, vdim=100)],
          [th.attention()], [th.attention(heads=3, kv_heads=1, dim=12, vdim=20, conv=4, window=64, dims=12, diff=0.7)],
          [th.attention(heads=2, kv_heads=2, dim=32, vdim=8, conv=1, window=130, dims=32)], [th.attention(heads=1, kv_heads=1, dim=8, vdim=8, conv=2, window=1, dims=0, diff=0.0)],
          [th.attention(heads=4, kv_heads=1, dim=64, vdim=128, conv=16, window=65, dims=32)], [th.attention(heads=2, kv_heads=1, dim=80, vdim=136, window=2, dims=80)],
          [th.latent(), th.latent(heads=5, dim=8, vdim=16, kv_from=0, scale=0.5), th.latent(heads=1, dim=12, vdim=10, kv_from=0)],
          [th.latent(heads=2, dim=12, rot_dim=4, vdim=10, rank=24), th.latent(heads=4, dim=24, rot_dim=4, vdim=8, rank=24, kv_from=0)],
          [th.latent(heads=1, dim=8, rot_dim=8, vdim=8, rank=8), th.latent(heads=17, dim=40, rot_dim=8, vdim=72, rank=8, kv_from=0)],
          [th.latent(heads=4, dim=64, rot_dim=32, vdim=64, rank=64), th.latent(heads=2, dim=96, rot_dim=32, vdim=136, rank=64, kv_from=0)]]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layers", LAYERS)
def test_mixers_alone(layers, dtype):
    """Prompts of unequal lengths in one step (one crossing pages and chunks, one of a single token), then tokens one by one;
    the same cut into portions, down to two tokens; then again in slots and pages that were used before."""
    w = th.draw_weights(th.config([(l, None) for l in layers], width=WIDTH), 6)
    rng = np.random.default_rng(7)
    lens, extra = [230, 20, 4, 1], 9
    xs = [pz.round_bf16(rng.standard_normal((n + extra, WIDTH))) for n in lens]
    refs = oracle(layers, xs, w, dtype == torch.bfloat16)
    mixers = Mixers(layers, dtype, w, sum(lens) + 4 * extra, 4, max(lens) + extra)
    for plan in ([lens] + [[1] * 4] * extra, [[2, 2, 2, 2], [100, 3, 3, 1], [137, 24, 8, 7]], [[n + extra for n in lens]]):
        for per, want in zip(mixers.run(xs, plan), refs):
            for g, r in zip(per, want):
                assert close(g, r, dtype), plan[0]


@pytest.mark.parametrize("change", ["gate", "difference", "convolution", "bias", "shared rows", "input gate", "output gate"])
def test_a_mechanism_left_out_shows(change):
    """The oracle itself moves by far more than the tolerance when a part of a mixer is left out or another layer's is used."""
    layers = {"shared rows": [th.latent(), th.latent(heads=5, dim=8, vdim=16, kv_from=0)], "input gate": [th.memory()], "output gate": [th.memory()]}.get(change, [th.attention()])
    w = th.draw_weights(th.config([(l, None) for l in layers], width=WIDTH), 6)
    xs = [pz.round_bf16(np.random.default_rng(7).standard_normal((100, WIDTH)))]
    px, other = "l0.mix.", dict(w)
    if change == "gate":
        other[px + "g"] = 0 * w[px + "g"]
    elif change == "difference":
        other[px + "lq1"] = w[px + "lq1"] + w[px + "lk1"]
    elif change == "convolution":
        other[px + "v.conv"] = w[px + "v.conv"][:, ::-1]
    elif change == "bias":
        other[px + "k.b"] = 0 * w[px + "k.b"]
    elif change == "shared rows":
        other[px + "dkv"] = -w[px + "dkv"][::-1]
    elif change == "input gate":
        other[px + "i"] = 0 * w[px + "i"]
    else:
        other[px + "g"] = 0 * w[px + "g"]
    a, b = oracle(layers, xs, w, False)[-1][0], oracle(layers, xs, other, False)[-1][0]
    assert np.sqrt(np.mean((a - b) ** 2)) > 3 * BF16_RMS_TOL * np.sqrt(np.mean(a ** 2))


@pytest.mark.parametrize("window", [1, 2, 63, 64, 65, 100])
def test_window_edges_show(window):
    """A large score scale makes each softmax pick almost one key, so a window that is one token off picks another one: in a
    prompt that crosses two page borders, cut there, and in the tokens decoded after it."""
    layer = th.attention(heads=2, kv_heads=1, dim=16, vdim=16, conv=2, window=window, scale=4.0)
    w = th.draw_weights(th.config([(layer, None)], width=WIDTH), 8)
    x = pz.round_bf16(np.random.default_rng(9).standard_normal((170, WIDTH)))
    a = pz.attention(x, layer["mixer"], w, "l0.mix.", EPS)
    for wrong in (window - 1, window + 1):
        if wrong:
            b = pz.attention(x, {**layer["mixer"], "mask": {"size": wrong}}, w, "l0.mix.", EPS)
            assert np.abs(a - b).max() > 1000 * FP32_TOL * np.abs(a).max()
    mixers = Mixers([layer], torch.float32, w, 170, 1, 170)
    for plan in ([[170]], [[150]] + [[1]] * 20, [[63], [2], [63], [42]]):
        assert close(mixers.run([x], plan)[0][0], a, torch.float32), plan[0]


def test_whole_prompts_of_latents_take_the_tensor_cores(monkeypatch):
    """bfloat16 prompts that start their sequences go through the tensor-core kernel, in the layer that owns the rows and in
    the one that reads them; the results agree with the kernel that scores the latents themselves."""
    from questwend_b200.parts import latent_attention as la
    layers = [th.latent(heads=3, dim=24, rot_dim=8, vdim=40), th.latent(heads=2, dim=40, rot_dim=8, vdim=16, kv_from=0)]
    w = th.draw_weights(th.config([(l, None) for l in layers], width=WIDTH), 10)
    xs = [pz.round_bf16(np.random.default_rng(n).standard_normal((n, WIDTH))) for n in (150, 64, 20, 1)]
    calls, kernel = [], ops.latent_prefill
    monkeypatch.setattr(ops, "latent_prefill", lambda *a, **k: calls.append(1) or kernel(*a, **k))
    mixers = Mixers(layers, torch.bfloat16, w, 400, 4, 200)
    got = mixers.run(xs, [[150, 64, 20, 1]])
    assert len(calls) == 2
    monkeypatch.setattr(la, "PROMPT_KERNEL_MIN_TOKENS", 10 ** 9)
    plain = mixers.run(xs, [[150, 64, 20, 1]])
    assert len(calls) == 2
    for per, other, want in zip(got, plain, oracle(layers, xs, w, True)):
        for g, p, r in zip(per, other, want):
            assert close(g, r, torch.bfloat16) and close(p, r, torch.bfloat16) and np.sqrt(np.mean((g - p) ** 2)) <= 0.02 * np.sqrt(np.mean(r ** 2))


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_keys_the_first_tokens_and_page_borders(dtype):
    """700 tokens of which some point away from another token hundreds of positions back, at the sequence's first positions, or
    at a page's first and last row, in latent attention (of its own rows, and of another layer's): whole, cut right there, and
    decoded.  Every head's queries point away from where the token's own key points, so such a query's weight goes to that
    other key; positions are not turned."""
    T, width = 700, 64
    layers = [th.latent(heads=2, dim=56, rot_dim=0, vdim=24, rank=64, scale=0.5), th.latent(heads=3, dim=40, rot_dim=0, vdim=16, rank=64, scale=0.7, kv_from=0)]
    w = th.draw_weights(th.config([(l, None) for l in layers], width=width), 9)
    for i in range(2):                                      # q = -W_uk W_dkv h, up to the latent's norm
        w[f"l{i}.mix.q"] = -pz.round_bf16(w[f"l{i}.mix.uk"] @ (w["l0.mix.dkv.norm"][:, None] * w["l0.mix.dkv"]))
    x = np.random.default_rng(10).standard_normal((T, width))
    pairs = [(T - 1, 70), (650, 127), (300, 0), (690, 1), (500, 448), (660, 63), (640, 64), (191, 128), (65, 2), (20, 3)]
    for query, key in pairs:
        x[query] = -3.0 * x[key]
    x = pz.round_bf16(x)
    refs = oracle(layers, [x], w, dtype == torch.bfloat16)
    for query, key in pairs:
        gone = x.copy()
        gone[key] = -gone[key]
        for ref, moved in zip(refs, oracle(layers, [gone[:query + 1]], w, False)):
            assert np.abs(ref[0][query] - moved[0][query]).max() > 0.2 * np.abs(ref[0][query]).max(), query
    rows = [q for q, _ in pairs]
    mixers = Mixers(layers, dtype, w, T, 1, T, width=width)
    for plan in ([[T]], [[640]] + [[1]] * 60, [[299], [2], [399]], [[64]] * 10 + [[2]] * 30):
        for per, ref in zip(mixers.run([x], plan), refs):
            assert close(per[0], ref[0], dtype), plan[0]
            assert np.abs(per[0][rows] - ref[0][rows]).max() <= 0.1 * np.abs(ref[0][rows]).max(), plan[0]


# ----------------------------------------------------------------------------- whole models
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, cfgd, seed in (("mixed", th.MIXED, 21), ("ones", th.ONES, 22)):
        w = th.draw_weights(cfgd, seed)
        out[name] = (th.write_folder(str(tmp_path_factory.mktemp(name)), cfgd, w), cfgd, w)
    return out


def all_rows(eng, slot, tokens):
    return host(eng.step([StepEntry(slot, list(tokens), list(range(len(tokens))))]))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", ["mixed", "ones"])
def test_model_whole_in_batches_in_portions_and_decoded(models, which, dtype):
    folder, cfgd, w = models[which]
    td = torch.float32 if dtype == "float32" else torch.bfloat16
    eng = Engine.from_folder(folder, dtype=dtype, max_tokens=2048, max_batch=4)
    seqs, refs = zip(*(th.clear_choices(cfgd, w, n, 31 + n, round16=td == torch.bfloat16) for n in (150, 1, 7, 66)))
    alone = []
    for t, ref in zip(seqs, refs):                          # each alone, whole
        (s,) = eng.open_sequences(1)
        alone.append(all_rows(eng, s, t))
        eng.close_sequences([s])
        assert rows_close(alone[-1], ref, td)
    # all in one batch of unequal lengths, in slots and pages that were used before: the same as alone
    slots = eng.open_sequences(4)
    out = host(eng.step([StepEntry(s, t, list(range(len(t)))) for s, t in zip(slots, seqs)]))
    eng.close_sequences(slots)
    off = 0
    for t, ref, one in zip(seqs, refs, alone):
        assert rows_close(out[off:off + len(t)], ref, td)
        if td == torch.float32:
            assert np.abs(out[off:off + len(t)] - one).max() <= FP32_TOL * np.abs(ref).max()
        off += len(t)
    # portions of several sizes, down to two tokens, in slots that were used before
    (s,) = eng.open_sequences(1)
    rows, at = [], 0
    for n in (2, 3, 60, 2, 17, 64, 2):
        rows.append(all_rows(eng, s, seqs[0][at:at + n]))
        at += n
    assert at == 150 and rows_close(np.concatenate(rows), refs[0], td)
    eng.close_sequences([s])
    # prompts cut at unequal places, then token by token together; the shorter ones end earlier and give their slots back
    cuts = [60, 1, 3, 8]
    slots = eng.open_sequences(4)
    rows = {i: [] for i in range(4)}
    first = host(eng.step([StepEntry(s, t[:c], list(range(c))) for s, t, c in zip(slots, seqs, cuts)]))
    off = 0
    for i, c in enumerate(cuts):
        rows[i] += list(first[off:off + c])
        off += c
    pos, live = list(cuts), [i for i in range(4) if cuts[i] < len(seqs[i])]
    eng.close_sequences([slots[i] for i in range(4) if i not in live])
    while live:
        out = host(eng.step([StepEntry(slots[i], [seqs[i][pos[i]]], [0]) for i in live]))
        for r, i in enumerate(live):
            rows[i].append(out[r])
            pos[i] += 1
        done = [i for i in live if pos[i] == len(seqs[i])]
        eng.close_sequences([slots[i] for i in done])
        live = [i for i in live if i not in done]
    for i, ref in enumerate(refs):
        assert rows_close(np.stack(rows[i]), ref, td), i
    assert eng.cache.slots.n_free == eng.max_batch and eng.cache.free_pages() == [g.pool.n for g in eng.cache._groups]


def test_layer_by_layer(models):
    """The stream after every scheduled layer against the plain implementation."""
    folder, cfgd, w = models["mixed"]
    eng = Engine.from_folder(folder, dtype="float32", max_tokens=512, max_batch=2)
    tokens, _ = th.clear_choices(cfgd, w, 90, 29, margin=1e-4)
    want = []
    pz.forward(cfgd, w, tokens, taps=want)
    (s,) = eng.open_sequences(1)
    ctx, rows = eng.build_context([StepEntry(s, tokens, [0])])
    got = []
    eng.model.forward(ctx, eng.unit_caches, rows, tap=lambda i, h: got.append(host(h)))
    assert len(got) == len(want) == len(cfgd["layers"])
    for g, r in zip(got, want):
        assert np.abs(g - r).max() <= FP32_TOL * np.abs(r).max()


def test_long_decoding_over_page_borders_and_windows(models):
    folder, cfgd, w = models["mixed"]
    eng = Engine.from_folder(folder, dtype="float32", max_tokens=512, max_batch=2)
    tokens, ref = th.clear_choices(cfgd, w, 280, 19, margin=1e-4)
    (s,) = eng.open_sequences(1)
    rows = list(all_rows(eng, s, tokens[:2]))
    for t in tokens[2:]:
        rows.append(host(eng.step([StepEntry(s, [t], [0])]))[0])
    assert close(np.stack(rows), ref, torch.float32)


def test_a_wide_model_with_many_rows(tmp_path):
    """Width 1,024 and a prompt of 600 tokens in bfloat16 (the sizes from which the products change kernels), then single
    tokens, and a batch of 20 single tokens."""
    cfgd = th.config([(th.attention(heads=4, kv_heads=2, dim=32, vdim=64, window=200, dims=32, scale=0.2), th.moe(ff=72, experts=8, top=3, shared=136)),
                      (th.memory(heads=2, dim=64, vdim=128, cap=8.0), th.moe(ff=40, experts=4, top=4, shared=264)),
                      (th.latent(heads=4, dim=64, rot_dim=32, vdim=64, rank=128, scale=0.1), None),
                      (th.latent(heads=2, dim=32, rot_dim=32, vdim=128, rank=128, scale=0.1, kv_from=2), None)], width=1024, vocab=128)
    w = th.draw_weights(cfgd, 41)
    folder = th.write_folder(str(tmp_path / "m"), cfgd, w)
    tokens = np.random.default_rng(3).integers(0, 128, 606).tolist()
    ref = pz.forward(cfgd, w, tokens, round16=True)
    eng = Engine.from_folder(folder, dtype="bfloat16", max_tokens=4096, max_batch=24, max_seq_len=700)
    (s,) = eng.open_sequences(1)
    rows = list(all_rows(eng, s, tokens[:600]))
    for t in tokens[600:]:
        rows.append(host(eng.step([StepEntry(s, [t], [0])]))[0])
    eng.close_sequences([s])
    assert rows_close(np.stack(rows), ref, torch.bfloat16)
    slots = eng.open_sequences(20)
    out = host(eng.step([StepEntry(s, tokens[i:i + 3], [2]) for i, s in enumerate(slots)]))
    out2 = host(eng.step([StepEntry(s, [tokens[i + 3]], [0]) for i, s in enumerate(slots)]))
    want = [pz.forward(cfgd, w, tokens[i:i + 4], round16=True) for i in range(20)]
    assert rows_close(out, np.stack([r[2] for r in want]), torch.bfloat16)
    assert rows_close(out2, np.stack([r[3] for r in want]), torch.bfloat16)


def test_memories_that_last_through_a_whole_model(tmp_path):
    """Forget gates near 1 in every matrix memory: a change of the first tokens still moves the logits 300 tokens later, and the
    engine, which decodes the last of them, follows."""
    cfgd = th.config([(th.memory(heads=2, dim=16, vdim=24), None), (th.memory(heads=3, dim=8, vdim=8), None)], width=48, vocab=50)
    w = th.draw_weights(cfgd, 12, lasting=True)
    folder = th.write_folder(str(tmp_path / "m"), cfgd, w)
    tokens = np.random.default_rng(4).integers(0, 50, 330).tolist()
    eng = Engine.from_folder(folder, dtype="float32", max_tokens=1024, max_batch=2)
    last = []
    for by in (0, 7):
        t = [(x + by) % 50 for x in tokens[:20]] + tokens[20:]
        ref = pz.forward(cfgd, w, t)
        (s,) = eng.open_sequences(1)
        rows = [all_rows(eng, s, t[:300])] + [host(eng.step([StepEntry(s, [x], [0])])) for x in t[300:]]
        eng.close_sequences([s])
        assert close(np.concatenate(rows), ref, torch.float32)
        last.append(ref[-1])
    assert np.abs(last[0] - last[1]).max() > 10 * FP32_TOL * np.abs(last[0]).max()


def test_generation_through_the_library_loop(models):
    """Greedy generation with the engine's own loop, scheduler, device sampler and CUDA graphs: two batches in slots that
    are used again, one request ending early, decoding across a page border; every chosen token is the plain
    implementation's choice."""
    import questwend_b200 as qw
    folder, cfgd, w = models["mixed"]
    eng = Engine.from_folder(folder, dtype="float32", max_tokens=1024, max_batch=3)
    rng = np.random.default_rng(17)
    prompts = [rng.integers(0, cfgd["vocab"], n).tolist() for n in (20, 1, 58, 5)]
    n_new = 24
    for use_graph in (True, False):
        free = qw.generate(eng, prompts, max_new_tokens=n_new, use_graph=use_graph)
        stop = free[2].tokens[6]
        stats = qw.GenerationStats()
        res = qw.generate(eng, prompts, max_new_tokens=n_new, stop_ids=[stop], use_graph=use_graph, stats=stats)
        assert stats.batches == 2 and res[2].finish_reason == "stop" and len(res[2].tokens) <= 7
        for run in (free, res):
            for p, r in zip(prompts, run):
                ref = pz.forward(cfgd, w, p + r.tokens)
                scale = np.abs(ref).max()
                for j, tok in enumerate(r.tokens):
                    row = ref[len(p) - 1 + j]
                    assert row.max() - row[tok] <= 2 * FP32_TOL * scale, (len(p), j, tok, int(row.argmax()))
    assert eng.cache.slots.n_free == eng.max_batch


def test_trace_replay_and_command_line(models, tmp_path):
    import os
    import subprocess
    import sys
    from helpers import ROOT
    folder, cfgd, w = models["ones"]
    V = cfgd["vocab"]
    rng = np.random.default_rng(23)
    a, b = rng.integers(0, V, 9).tolist(), rng.integers(0, V, 4).tolist()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:7], "want": [0, 6]}, {"id": "b", "tokens": b[:3], "want": [2]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[7:8], "want": []}, {"id": "b", "tokens": b[3:], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[8:], "want": [0]}], "end": ["a"]}]
    out = run_trace(folder, "float32", steps, 256, str(tmp_path / "out"))
    ra, rb = pz.forward(cfgd, w, a), pz.forward(cfgd, w, b)
    assert close(out[0], np.stack([ra[0], ra[6], rb[2]]), torch.float32)
    assert close(out[1], rb[3:4], torch.float32) and close(out[2], ra[8:9], torch.float32)
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "qw-cli"), "-m", folder, "-p", " ".join(map(str, a)),
                           "-n", "5", "--dtype", "float32"], capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr
    ids = [int(x) for x in proc.stdout.split()]
    ref = pz.forward(cfgd, w, a + ids)
    for j, tok in enumerate(ids):
        row = ref[len(a) - 1 + j]
        assert row.max() - row[tok] <= 2 * FP32_TOL * np.abs(ref).max()
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "qw-cli"), "-m", folder, "--info"], capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0 and "Tebozen" in proc.stdout
