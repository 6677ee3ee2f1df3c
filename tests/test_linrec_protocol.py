"""Simulation of the hand-offs inside the tcgen05 recurrence kernel (csrc/tkv_linrec_tc.cu) under random interleavings.

Each role of a CTA is a generator that performs one action at a time (two generators stand for the threads of a row role, so
that they can drift apart); copies and products complete asynchronously, products of one issuing thread in order.  Barriers
behave like mbarriers: a wait names a parity, returns when the phase of that parity is the last one completed, and cannot tell
a phase from the one two later.  Checked: nobody waits for good, no wait returns before the phase it means, every read finds
the chunk it expects, and nothing is overwritten while a product reads it.
"""
import random

import pytest


class Bar:
    def __init__(self, count):
        self.count, self.pending, self.phase = count, count, 0      # phase: index of the one in progress

    def arrive(self):
        self.pending -= 1
        if self.pending == 0:
            self.phase, self.pending = self.phase + 1, self.count


class Sim:
    def __init__(self, nchunks, state_only, partial, rng):
        self.n, self.so, self.partial, self.rng = nchunks, state_only, partial, rng
        two = 2
        self.bar = {k: Bar(1) for k in ("qk", "v0", "v1", "l0", "l1", "s", "o1", "st", "o2")}
        self.bar.update({k: Bar(two) for k in ("sp", "wv", "p", "clr")})
        self.buf = {}                                               # resource -> chunk it holds
        self.busy = {}                                              # resource -> products reading it
        self.queues = {"main": [], "tma": []}

    # ---- primitives
    def wait(self, name, phase):
        while (self.bar[name].phase & 1) == (phase & 1):
            yield ("wait", name, phase)
        assert self.bar[name].phase == phase + 1, f"wait for phase {phase} of {name} returned in phase {self.bar[name].phase}"

    def write(self, res, chunk):
        assert not self.busy.get(res), f"{res} overwritten with chunk {chunk} while a product reads it"
        self.buf[res] = chunk

    def read(self, res, chunk):
        assert self.buf.get(res) == chunk, f"{res} holds {self.buf.get(res)}, chunk {chunk} expected"

    def product(self, queue, reads, out, chunk, bar):
        for r in reads:
            self.read(r, chunk)
            self.busy[r] = self.busy.get(r, 0) + 1
        self.write(out, ("writing", chunk))
        self.queues[queue].append((reads, out, chunk, bar))

    def copy(self, res, chunk, bar):
        for r in res:
            self.write(r, ("loading", chunk))
        self.queues["tma"].append((res, None, chunk, bar))

    def complete(self, queue):
        q = self.queues[queue]
        reads, out, chunk, bar = q.pop(self.rng.randrange(len(q)) if queue == "tma" else 0)
        if queue == "tma":
            for r in reads:
                self.buf[r] = chunk
        else:
            for r in reads:
                self.busy[r] -= 1
            self.buf[out] = chunk
        if bar is not None:
            self.bar[bar].arrive()

    # ---- roles
    def load_qk(self, i):
        self.copy(["K"] if self.so else ["Q", "K"], i, "qk")

    def load_v(self, i):
        self.copy([f"V{i & 1}"], i, f"v{i & 1}")

    def control(self):
        self.load_qk(0)
        self.load_v(0)
        for i in range(self.n):
            yield from self.wait("qk", i)
            if i == self.n - 1 and self.partial:
                yield from self.wait("clr", 0)
            if not self.so:
                self.product("main", ["Q", "K"], "S", i, "s")
                yield
            yield from self.wait("sp", i)
            if i + 1 < self.n:
                self.load_v(i + 1)
            if not self.so:
                self.product("main", ["Q", "SP"], "O1", i, "o1")
                yield
            yield from self.wait("wv", i)
            self.product("main", ["K", "WV"], "ST", i, "st")
            yield
            if i + 1 < self.n:
                yield from self.wait("st", i)
                if not self.so:
                    yield from self.wait("o1", i)
                self.load_qk(i + 1)
                yield
            if not self.so:
                yield from self.wait("p", i)
                self.product("main", ["P", f"V{i & 1}"], "O2", i, "o2")
                yield

    def scan(self):
        for i in range(self.n):
            if i >= 1:
                yield from self.wait("sp", i - 1)
            self.write(f"L{i & 1}", i)
            yield
            self.bar[f"l{i & 1}"].arrive()
            yield

    def rows(self):
        for i in range(self.n):
            if i == self.n - 1 and self.partial:
                yield from self.wait("qk", i)
                yield from self.wait(f"v{i & 1}", i >> 1)
                self.write("K", i)
                self.write(f"V{i & 1}", i)
                yield
                self.bar["clr"].arrive()
                yield
            yield from self.wait(f"l{i & 1}", i >> 1)
            if i > 0:
                yield from self.wait("st", i - 1)
                self.read("ST", i - 1)
            self.read(f"L{i & 1}", i)
            if not self.so:
                self.write("SP", i)
                yield
            self.bar["sp"].arrive()
            yield
            yield from self.wait(f"v{i & 1}", i >> 1)
            self.read(f"V{i & 1}", i)
            self.read(f"L{i & 1}", i)
            self.write("WV", i)
            yield
            self.bar["wv"].arrive()
            yield
            if self.so:
                continue
            yield from self.wait("s", i)
            for _ in range(2):
                self.read("S", i)
                self.read(f"L{i & 1}", i)
                self.write("P", i)
                yield
            self.bar["p"].arrive()
            yield
            yield from self.wait("o1", i)
            yield from self.wait("o2", i)
            for res in ("O1", "O2", f"V{i & 1}", f"L{i & 1}"):
                self.read(res, i)
                yield
        yield from self.wait("st", self.n - 1)
        self.read("ST", self.n - 1)

    def agents(self):
        return [self.control(), self.scan(), self.rows(), self.rows()]

    def run(self):
        agents = self.agents()
        speed = [self.rng.choice([1, 1, 4, 30]) for _ in agents]
        blocked = {}
        while agents:
            pending = [q for q in self.queues if self.queues[q]]
            live = [k for k in range(len(agents)) if not (k in blocked and (self.bar[blocked[k][0]].phase & 1) == (blocked[k][1] & 1))]
            assert live or pending, f"everyone waits: {blocked}"
            if pending and (not live or self.rng.random() < 0.2):
                self.complete(self.rng.choice(pending))
                continue
            k = self.rng.choices(live, [speed[x] for x in live])[0]
            try:
                y = next(agents[k])
                blocked.pop(k, None)
                if y is not None:
                    blocked[k] = y[1:]
            except StopIteration:
                agents.pop(k)
                speed.pop(k)
                blocked = {(x if x < k else x - 1): v for x, v in blocked.items() if x != k}


@pytest.mark.parametrize("state_only", [False, True])
@pytest.mark.parametrize("nchunks", [1, 2, 3, 4, 9])
def test_hand_offs_hold_under_random_interleavings(nchunks, state_only):
    for seed in range(200):
        rng = random.Random(1000 * nchunks + seed)
        Sim(nchunks, state_only, partial=not state_only and bool(seed & 1), rng=rng).run()


def test_the_simulation_notices_a_missing_wait():
    """With the wait for the previous state update taken out of the model, some interleaving overwrites what it reads."""
    class Broken(Sim):
        def wait(self, name, phase):
            if name == "st":
                return
            yield from super().wait(name, phase)
    with pytest.raises(AssertionError):
        for seed in range(300):
            Broken(6, False, False, random.Random(seed)).run()
