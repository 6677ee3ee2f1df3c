"""Simulation of the hand-offs inside the tcgen05 kernel of the channel-decay recurrence (csrc/tkv_chanrec_tc.cu) under random
interleavings, with the barriers and checks of ``test_linrec_protocol``: nobody waits for good, no wait returns before the phase
it means, every read finds the chunk it expects, and nothing is overwritten while a product reads it."""
import random

import pytest

from tests.test_linrec_protocol import Bar, Sim


class ChanSim(Sim):
    def __init__(self, nchunks, state_only, rng):
        super().__init__(nchunks, state_only, False, rng)
        self.bar = {k: Bar(1) for k in ("done0", "done1")}
        self.bar.update({k: Bar(2) for k in ("full0", "full1", "sop", "sync0", "sync1", "sync2")})

    def agents(self):
        return [self.gates(0), self.gates(1), self.state(True), self.state(False)]

    def products(self, i):
        self.product("main", [f"K{i & 1}", f"V{i % 3}"], "ST", i, f"done{i & 1}" if self.so else None)
        if not self.so:
            self.product("main", [f"Q{i & 1}", f"A{i & 1}", f"V{i % 3}", "SOP"], f"O{i & 1}", i, f"done{i & 1}")

    def meet(self, which, i):
        self.bar[f"sync{which}"].arrive()
        yield
        yield from self.wait(f"sync{which}", i)

    def gates(self, k):
        def load(i):                                                # each thread copies its own part and waits for it itself
            self.write(f"raw{i & 1}.{k}", ("loading", i))
            self.write(f"V{i % 3}", i)

        def see(i):
            for part in (0, 1):
                self.read(f"raw{i & 1}.{part}", i)
        load(0)
        for i in range(self.n):
            if i >= 2:
                yield from self.wait(f"done{i & 1}", (i - 2) >> 1)
            self.buf[f"raw{i & 1}.{k}"] = i
            yield
            yield from self.meet(0, i)
            if i + 1 < self.n:
                load(i + 1)
            yield
            see(i)
            self.write(f"oct.{k}", i)
            yield
            yield from self.meet(1, i)
            for part in (0, 1):
                self.read(f"oct.{part}", i)
            see(i)
            yield
            self.write(f"K{i & 1}", i)
            if not self.so:
                self.write(f"Q{i & 1}", i)
                self.write(f"QH.{k}", i)
                yield
                yield from self.meet(2, i)
                for part in (0, 1):
                    self.read(f"QH.{part}", i)
                see(i)                                              # (the pair-by-pair form reads the projections again)
                self.write(f"A{i & 1}", i)
                yield
                for part in (0, 1):
                    self.read(f"QH.{part}", i)
            yield
            self.bar[f"full{i & 1}"].arrive()
            yield

    def state(self, issues):
        for i in range(self.n):
            if i > 0:
                yield from self.wait(f"done{(i - 1) & 1}", (i - 1) >> 1)
                self.read("ST", i - 1)
            yield from self.wait(f"full{i & 1}", i >> 1)
            self.read(f"K{i & 1}", i)                               # stands for the chunk's factors of the state
            if not self.so:
                self.write("SOP", i)
            yield
            if i > 0:
                self.read("ST", i - 1)
            self.bar["sop"].arrive()
            yield
            if issues:
                yield from self.wait("sop", i)
                self.products(i)
                yield
            if i > 0 and not self.so:
                self.read(f"O{(i - 1) & 1}", i - 1)
                yield
                self.read(f"O{(i - 1) & 1}", i - 1)
        yield from self.wait(f"done{(self.n - 1) & 1}", (self.n - 1) >> 1)
        self.read("ST", self.n - 1)


@pytest.mark.parametrize("state_only", [False, True])
@pytest.mark.parametrize("nchunks", [1, 2, 3, 4, 9])
def test_hand_offs_hold_under_random_interleavings(nchunks, state_only):
    for seed in range(200):
        ChanSim(nchunks, state_only, random.Random(1000 * nchunks + seed)).run()


@pytest.mark.parametrize("missing", ["done0", "sop", "sync0"])
def test_the_simulation_notices_a_missing_wait(missing):
    class Broken(ChanSim):
        def wait(self, name, phase):
            if name == missing:
                return
            yield from super().wait(name, phase)
    with pytest.raises(AssertionError):
        for seed in range(300):
            Broken(6, False, random.Random(seed)).run()
