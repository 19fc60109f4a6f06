"""name -> factory tables (utils/registry.py:6-40)."""
from __future__ import annotations


class Registry:
    def __init__(self, kind: str):
        self._kind, self._items = kind, {}

    def register(self, name: str):
        if name in self._items:
            raise KeyError(f"{self._kind} '{name}' is already registered.")

        def decorator(item):
            self._items[name] = item
            return item
        return decorator

    def __getitem__(self, name: str):
        if name not in self._items:
            raise KeyError(f"Unsupported {self._kind}: {name}")
        return self._items[name]

    def supported_names(self):
        return list(self._items)
