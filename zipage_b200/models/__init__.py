"""Models that the serving loop runs, chosen by a folder's config.json (`registry.load_model`)."""
